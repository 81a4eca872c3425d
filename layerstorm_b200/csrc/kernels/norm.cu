// RMSNorm family and the hyper-connection (mHC) residual-stream kernels.
//
// RMSNorm: plain, strided, fused residual add (reference: src/compute/kernels/sm120/norm/rmsnorm.cu:71-164).
// mHC: `hc_mult` residual streams per token; "pre" mixes them into the sublayer input
// (sigmoid gates, Sinkhorn-normalised stream-mixing matrix), "post" writes the sublayer
// output back (reference: launchers in src/compute/kernels/mhc/mhc.h, math in
// tools/glm53_numpy_ref.py:128-179).  Here post of sublayer i and pre of sublayer i+1
// are one fused pass: a partial kernel spread over the hidden dimension followed by a
// one-block-per-token finalize that also applies the sublayer's input RMSNorm.
#include "common.cuh"
#include "comm.cuh"

namespace lsb {

template <typename TIn>
__device__ __forceinline__ float ld_as_float(const TIn* p, int i);
template <>
__device__ __forceinline__ float ld_as_float<float>(const float* p, int i) { return p[i]; }
template <>
__device__ __forceinline__ float ld_as_float<bf16>(const bf16* p, int i) { return __bfloat162float(p[i]); }

// out[r] = x[r] / sqrt(mean(x[r]^2) + eps) * w ; optional: resid[r] += x[r] first and
// normalise the sum (resid updated in place, fp32).
template <typename TIn, bool ADD>
__global__ void rmsnorm_kernel(bf16* __restrict__ out, const TIn* __restrict__ x, float* __restrict__ resid,
                               const float* __restrict__ w, int dim, int ldx, int ldo, int ldr, float eps,
                               float* __restrict__ out_f32, PeerComm comm) {
    __shared__ float red[33];
    extern __shared__ float row[];
    const int r = blockIdx.x;
    const TIn* xr = x + (size_t)r * ldx;
    pdl_wait();
    pdl_launch_dependents();
    unsigned epoch = 0;
    if (comm.nranks) {
        epoch = *comm.epoch;
        if (comm.xchg) {
            // consumer-side exchange: this block ships its row of the local partial to the peers, then waits for theirs
            for (int i = threadIdx.x; i < dim; i += blockDim.x) {
                const float v = ld_as_float<TIn>(xr, i);
                if (comm.xchg == 2) comm_ll_put<1>(comm, epoch, (size_t)r * ldx + i, &v);
                else comm_xchg_put<1>(comm, epoch, (size_t)r * ldx + i, &v);
            }
            if (comm.xchg != 2) comm_xchg_sync(comm, epoch, r);
        } else {
            comm_wait(comm, epoch);
        }
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float v;
        if (comm.nranks && comm.xchg == 2) { const float own = ld_as_float<TIn>(xr, i); comm_ll_get<1>(comm, epoch, (size_t)r * ldx + i, &own, &v); }
        else v = comm.nranks ? (comm.xchg ? comm_xchg_get(comm, epoch, (size_t)r * ldx + i, ld_as_float<TIn>(xr, i)) : comm_reduce(comm, epoch, (size_t)r * ldx + i))
                             : ld_as_float<TIn>(xr, i);
        if (ADD) {
            v += resid[(size_t)r * ldr + i];
            resid[(size_t)r * ldr + i] = v;
        }
        row[i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)dim + eps);
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const float v = row[i] * inv * w[i];
        out[(size_t)r * ldo + i] = __float2bfloat16(v);
        if (out_f32) out_f32[(size_t)r * ldo + i] = v;
    }
    pdl_launch_dependents();
}

constexpr int kHcMax = 4;           // residual streams
constexpr int kHcOut = 2 * kHcMax + kHcMax * kHcMax;   // 24 mixing logits
constexpr int kHcChunk = 32;        // hidden columns per partial block
constexpr int kHcPerWarp = 6;       // mixing logits per warp (4 warps x 6 = 24)

// Pass 1 of post+pre.  mode 0: residual[j] = x (replicate, first layer);
// mode 1: residual[j] = post[j]*x + sum_i comb[i][j]*residual[i].
// Then partial mixing logits and partial sum of squares of the NEW residual over this
// block's 32 hidden columns: part[r][chunk][0..23] logits, [24] sum of squares.
// Lane = column, warp = a group of 6 mixing logits; every warp recomputes the (cheap) residual
// update, warp 0 stores it.
__global__ void __launch_bounds__(128) mhc_post_partial_kernel(float* __restrict__ residual, const float* __restrict__ x,
                                                               const float* __restrict__ post, const float* __restrict__ comb,
                                                               const float* __restrict__ fn, float* __restrict__ part,
                                                               int hidden, int n, int mode, int rows, int rows_per_block, PeerComm comm) {
    const int c = blockIdx.y, lane = threadIdx.x & 31, og = threadIdx.x >> 5;
    const int h = c * kHcChunk + lane;
    const int nout = 2 * n + n * n;
    // mixing-matrix rows do not depend on the previous kernel: fetch them before the dependency wait
    float f[kHcPerWarp][kHcMax];
#pragma unroll
    for (int i = 0; i < kHcPerWarp; ++i) {
        const int o = og * kHcPerWarp + i;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j) f[i][j] = (o < nout && j < n) ? __ldg(fn + ((size_t)o * n + j) * hidden + h) : 0.f;
    }
    pdl_wait();
    pdl_launch_dependents();
    unsigned epoch = 0;
    if (comm.nranks && mode == 1) {
        epoch = *comm.epoch;
        comm_wait(comm, epoch);
    }
    // a block serves `rows_per_block` consecutive rows with the same register-resident mixing rows
    for (int r = blockIdx.x * rows_per_block; r < min(rows, (int)(blockIdx.x + 1) * rows_per_block); ++r) {
        float res[kHcMax];
        float* rp = residual + (size_t)r * n * hidden;
        const float xv = (comm.nranks && mode == 1) ? comm_reduce(comm, epoch, (size_t)r * hidden + h) : x[(size_t)r * hidden + h];
        if (mode == 0) {
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) res[j] = j < n ? xv : 0.f;
        } else {
            float old[kHcMax];
#pragma unroll
            for (int i = 0; i < kHcMax; ++i) old[i] = i < n ? rp[(size_t)i * hidden + h] : 0.f;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) {
                float a = 0.f;
                if (j < n) {
                    a = post[r * n + j] * xv;
                    for (int i = 0; i < n; ++i) a += comb[(r * n + i) * n + j] * old[i];
                }
                res[j] = a;
            }
        }
        float* po = part + ((size_t)r * gridDim.y + c) * (kHcOut + 1);
#pragma unroll
        for (int i = 0; i < kHcPerWarp; ++i) {
            float a = 0.f;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) a = fmaf(res[j], f[i][j], a);
            a = warp_sum(a);
            const int o = og * kHcPerWarp + i;
            if (lane == 0 && o < kHcOut) po[o] = a;
        }
        __syncthreads();                              // every warp has read the old streams of this row (in-place update by warp 0)
        if (og == 0) {
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j)
                if (j < n) { rp[(size_t)j * hidden + h] = res[j]; ss += res[j] * res[j]; }
            ss = warp_sum(ss);
            if (lane == 0) po[kHcOut] = ss;
        }
    }
    pdl_launch_dependents();
}

// Many-row variant of the pass above: a block covers 128 hidden columns (4 consecutive columns per lane, 16-byte
// loads and stores), so the 25 warp reductions per (row, block) amortise over four times the columns - with 2048-row
// prefill chunks the narrow kernel is bound by its shuffles, not by memory.  part[r][chunk128][0..24].
constexpr int kHcWide = 128;
__global__ void __launch_bounds__(128) mhc_post_partial_wide_kernel(float* __restrict__ residual, const float* __restrict__ x,
                                                                    const float* __restrict__ post, const float* __restrict__ comb,
                                                                    const float* __restrict__ fn, float* __restrict__ part,
                                                                    int hidden, int n, int mode, int rows, int rows_per_block, PeerComm comm) {
    const int c = blockIdx.x, lane = threadIdx.x & 31, og = threadIdx.x >> 5;
    const int h = c * kHcWide + lane * 4;
    const int nout = 2 * n + n * n;
    float4 f[kHcPerWarp][kHcMax];
#pragma unroll
    for (int i = 0; i < kHcPerWarp; ++i) {
        const int o = og * kHcPerWarp + i;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j)
            f[i][j] = (o < nout && j < n) ? __ldg(reinterpret_cast<const float4*>(fn + ((size_t)o * n + j) * hidden + h)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    pdl_launch_dependents();
    unsigned epoch = 0;
    if (comm.nranks && mode == 1) {
        epoch = *comm.epoch;
        comm_wait(comm, epoch);
    }
    // The rows of a block are independent but each one is a chain load -> mix -> 7 warp reductions -> store: with one row in
    // flight the block waits a DRAM round trip per row (16 per block).  The next row's operands (x, the four old streams, its
    // post / comb gates: 10 16-byte loads) are therefore requested before the current row is worked on.
    struct RowIn { float4 xv; float4 old[kHcMax]; float pj[kHcMax]; float cj[kHcMax][kHcMax]; };
    const float4 z4 = make_float4(0.f, 0.f, 0.f, 0.f);
    auto load_row = [&](int r, RowIn& in) {
        const float* rp = residual + (size_t)r * n * hidden;
        if (comm.nranks && mode == 1) {
            const size_t b = (size_t)r * hidden + h;
            in.xv = make_float4(comm_reduce(comm, epoch, b), comm_reduce(comm, epoch, b + 1), comm_reduce(comm, epoch, b + 2), comm_reduce(comm, epoch, b + 3));
        } else {
            in.xv = *reinterpret_cast<const float4*>(x + (size_t)r * hidden + h);
        }
        if (mode != 0) {
#pragma unroll
            for (int i = 0; i < kHcMax; ++i) in.old[i] = i < n ? *reinterpret_cast<const float4*>(rp + (size_t)i * hidden + h) : z4;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) {
                in.pj[j] = j < n ? post[r * n + j] : 0.f;
#pragma unroll
                for (int i = 0; i < kHcMax; ++i) in.cj[i][j] = (i < n && j < n) ? comb[(r * n + i) * n + j] : 0.f;
            }
        }
    };
    const int r_begin = blockIdx.y * rows_per_block, r_end = min(rows, (int)(blockIdx.y + 1) * rows_per_block);
    RowIn cur, nxt;
    if (r_begin < r_end) load_row(r_begin, cur);
    for (int r = r_begin; r < r_end; ++r) {
        if (r + 1 < r_end) load_row(r + 1, nxt);      // (rows are disjoint: the in-place store of row r below never touches row r + 1)
        float4 res[kHcMax];
        float* rp = residual + (size_t)r * n * hidden;
        if (mode == 0) {
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) res[j] = j < n ? cur.xv : z4;
        } else {
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) {
                float4 a = z4;
                if (j < n) {
                    const float pj = cur.pj[j];
                    a = make_float4(pj * cur.xv.x, pj * cur.xv.y, pj * cur.xv.z, pj * cur.xv.w);
#pragma unroll
                    for (int i = 0; i < kHcMax; ++i) {
                        if (i < n) {
                            const float cj = cur.cj[i][j];
                            a.x += cj * cur.old[i].x; a.y += cj * cur.old[i].y; a.z += cj * cur.old[i].z; a.w += cj * cur.old[i].w;
                        }
                    }
                }
                res[j] = a;
            }
        }
        float* po = part + ((size_t)r * gridDim.x + c) * (kHcOut + 1);
#pragma unroll
        for (int i = 0; i < kHcPerWarp; ++i) {
            float a = 0.f;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) {
                a = fmaf(res[j].x, f[i][j].x, a); a = fmaf(res[j].y, f[i][j].y, a);
                a = fmaf(res[j].z, f[i][j].z, a); a = fmaf(res[j].w, f[i][j].w, a);
            }
            a = warp_sum(a);
            const int o = og * kHcPerWarp + i;
            if (lane == 0 && o < kHcOut) po[o] = a;
        }
        // the residual is updated in place by warp 0 while every warp of the block read the old streams of this row above:
        // all of them must have done so before the store (warps drift apart over the row loop)
        __syncthreads();
        if (og == 0) {
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j)
                if (j < n) {
                    *reinterpret_cast<float4*>(rp + (size_t)j * hidden + h) = res[j];
                    ss += res[j].x * res[j].x + res[j].y * res[j].y + res[j].z * res[j].z + res[j].w * res[j].w;
                }
            ss = warp_sum(ss);
            if (lane == 0) po[kHcOut] = ss;
        }
        cur = nxt;
    }
    pdl_launch_dependents();
}

// Pass 2: reduce the partials in a fixed order, form pre/post gates and the Sinkhorn-
// normalised mixing matrix (one matrix element per lane, sums by shuffles), then
// out = RMSNorm(sum_j pre[j]*residual[j]) * w (bf16).
__global__ void __launch_bounds__(512) mhc_finalize_kernel(bf16* __restrict__ out, const float* __restrict__ residual, const float* __restrict__ part,
                                                           const float* __restrict__ hc_scale, const float* __restrict__ hc_base,
                                                           const float* __restrict__ norm_w, float* __restrict__ post_out, float* __restrict__ comb_out,
                                                           int hidden, int n, int nchunks, int iters, float hc_eps, float rms_eps, float post_mult) {
    __shared__ float red[33];
    __shared__ float mix[kHcOut + 1];
    __shared__ float pre[kHcMax];
    extern __shared__ float row[];
    const int r = blockIdx.x, t = threadIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    {
        const int o = t >> 4, sub = t & 15;
        float a = 0.f;
        if (o <= kHcOut) {
            // batches of 8 independent loads: the adds must not serialise the memory latency
            for (int c0 = sub; c0 < nchunks; c0 += 128) {
                float v[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const int c = c0 + u * 16;
                    v[u] = c < nchunks ? part[((size_t)r * nchunks + c) * (kHcOut + 1) + o] : 0.f;
                }
#pragma unroll
                for (int u = 0; u < 8; ++u) a += v[u];
            }
        }
#pragma unroll
        for (int d = 8; d > 0; d >>= 1) a += __shfl_xor_sync(0xffffffffu, a, d, 16);
        if (sub == 0 && o <= kHcOut) mix[o] = a;
    }
    __syncthreads();
    if (t < 32) {
        const float inv = rsqrtf(mix[kHcOut] / (float)(n * hidden) + rms_eps);
        if (t < 16) {
            const int i = t >> 2, j = t & 3;
            const bool valid = i < n && j < n;
            float v = valid ? mix[2 * n + i * n + j] * inv * hc_scale[2] + hc_base[2 * n + i * n + j] : -INFINITY;
            float mx = fmaxf(v, __shfl_xor_sync(0xffffu, v, 1, 16));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffu, mx, 2, 16));
            float e = valid ? expf(v - mx) : 0.f;
            float s = e + __shfl_xor_sync(0xffffu, e, 1, 16);
            s += __shfl_xor_sync(0xffffu, s, 2, 16);
            float cm = valid ? e / s + hc_eps : 0.f;
            // column normalise, then (iters-1) x (row normalise, column normalise)
            float cs = cm + __shfl_xor_sync(0xffffu, cm, 4, 16);
            cs += __shfl_xor_sync(0xffffu, cs, 8, 16);
            cm = valid ? cm / (cs + hc_eps) : 0.f;
            for (int it = 1; it < iters; ++it) {
                float rs = cm + __shfl_xor_sync(0xffffu, cm, 1, 16);
                rs += __shfl_xor_sync(0xffffu, rs, 2, 16);
                cm = valid ? cm / (rs + hc_eps) : 0.f;
                cs = cm + __shfl_xor_sync(0xffffu, cm, 4, 16);
                cs += __shfl_xor_sync(0xffffu, cs, 8, 16);
                cm = valid ? cm / (cs + hc_eps) : 0.f;
            }
            if (valid) comb_out[(r * n + i) * n + j] = cm;
        } else if (t < 16 + kHcMax) {
            const int j = t - 16;
            if (j < n) pre[j] = sigmoidf_(mix[j] * inv * hc_scale[0] + hc_base[j]) + hc_eps;
        } else if (t < 16 + 2 * kHcMax) {
            const int j = t - 16 - kHcMax;
            if (j < n) post_out[r * n + j] = sigmoidf_(mix[n + j] * inv * hc_scale[1] + hc_base[n + j]) * post_mult;
        }
    }
    __syncthreads();
    const float* rp = residual + (size_t)r * n * hidden;
    float ss = 0.f;
    float pj[kHcMax];
#pragma unroll
    for (int j = 0; j < kHcMax; ++j) pj[j] = j < n ? pre[j] : 0.f;
    for (int h0 = t; h0 < hidden; h0 += blockDim.x * 4) {
        float v[4][kHcMax];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int h = h0 + u * blockDim.x;
#pragma unroll
            for (int j = 0; j < kHcMax; ++j) v[u][j] = (h < hidden && j < n) ? rp[(size_t)j * hidden + h] : 0.f;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int h = h0 + u * blockDim.x;
            if (h < hidden) {
                float a = 0.f;
#pragma unroll
                for (int j = 0; j < kHcMax; ++j) a += pj[j] * v[u][j];
                row[h] = a;
                ss += a * a;
            }
        }
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)hidden + rms_eps);
    for (int h = t; h < hidden; h += blockDim.x) out[(size_t)r * hidden + h] = __float2bfloat16(row[h] * inv * norm_w[h]);
    pdl_launch_dependents();
}


// ---- few-row (decode) variant: two launches instead of partial + one-block-per-row finalize -------------------------------
// mhc_post_fused: same residual update and partial mixing logits as mhc_post_partial, plus the partial Gram matrix
// G[j][j'] = sum_h res_j[h] res_j'[h] of the new residual streams.  The last block of a row to finish (atomic counter)
// reduces the partials in chunk order, forms pre / post and the Sinkhorn-normalised mixing matrix, and gets the RMS of the
// contracted vector algebraically:  sum_h (sum_j pre_j res_j[h])^2 = pre^T G pre  - no second pass over the hidden dimension.
// mhc_contract: out[h] = inv_rms * w[h] * sum_j pre_j res_j[h], fully parallel over the hidden dimension.
constexpr int kHcGram = kHcMax * (kHcMax + 1) / 2;         // 10
constexpr int kHcPart2 = kHcOut + kHcGram + 2;             // 36 floats per (row, chunk)

__global__ void __launch_bounds__(128) mhc_post_fused_kernel(float* __restrict__ residual, const float* __restrict__ x,
                                                             float* __restrict__ post, float* __restrict__ comb,
                                                             const float* __restrict__ fn, const float* __restrict__ hc_scale,
                                                             const float* __restrict__ hc_base, float* __restrict__ part,
                                                             unsigned* __restrict__ done, float* __restrict__ prex, int hidden, int n, int mode,
                                                             int iters, float hc_eps, float rms_eps, float post_mult, PeerComm comm) {
    __shared__ float mix[kHcPart2];
    __shared__ int s_last;
    const int r = blockIdx.x, c = blockIdx.y, lane = threadIdx.x & 31, og = threadIdx.x >> 5, t = threadIdx.x;
    const int nchunks = gridDim.y;
    const int h = c * kHcChunk + lane;
    const int nout = 2 * n + n * n;
    float f[kHcPerWarp][kHcMax];
#pragma unroll
    for (int i = 0; i < kHcPerWarp; ++i) {
        const int o = og * kHcPerWarp + i;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j) f[i][j] = (o < nout && j < n) ? __ldg(fn + ((size_t)o * n + j) * hidden + h) : 0.f;
    }
    pdl_wait();
    pdl_launch_dependents();
    float res[kHcMax];
    float* rp = residual + (size_t)r * n * hidden;
    float xv;
    if (comm.nranks && mode == 1) {
        const unsigned epoch = *comm.epoch;
        comm_wait(comm, epoch);
        xv = comm_reduce(comm, epoch, (size_t)r * hidden + h);
    } else {
        xv = x[(size_t)r * hidden + h];
    }
    if (mode == 0) {
#pragma unroll
        for (int j = 0; j < kHcMax; ++j) res[j] = j < n ? xv : 0.f;
    } else {
        float old[kHcMax];
#pragma unroll
        for (int i = 0; i < kHcMax; ++i) old[i] = i < n ? rp[(size_t)i * hidden + h] : 0.f;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j) {
            float a = 0.f;
            if (j < n) {
                a = post[r * n + j] * xv;
                for (int i = 0; i < n; ++i) a += comb[(r * n + i) * n + j] * old[i];
            }
            res[j] = a;
        }
    }
    float* po = part + ((size_t)r * nchunks + c) * kHcPart2;
#pragma unroll
    for (int i = 0; i < kHcPerWarp; ++i) {
        float a = 0.f;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j) a = fmaf(res[j], f[i][j], a);
        a = warp_sum(a);
        const int o = og * kHcPerWarp + i;
        if (lane == 0 && o < kHcOut) po[o] = a;
    }
    // Gram entries (j <= j'), spread over the four warps: warp w takes entries w, w+4, w+8
    {
        int e = 0;
#pragma unroll
        for (int j = 0; j < kHcMax; ++j)
#pragma unroll
            for (int k = j; k < kHcMax; ++k, ++e)
                if ((e & 3) == og) {
                    const float g = warp_sum(res[j] * res[k]);
                    if (lane == 0) po[kHcOut + e] = g;
                }
    }
    __syncthreads();                                  // every warp has read the old streams (in-place update by warp 0)
    if (og == 0) {
#pragma unroll
        for (int j = 0; j < kHcMax; ++j)
            if (j < n) rp[(size_t)j * hidden + h] = res[j];
    }
    // ---- last block of this row finishes the job ----
    __threadfence();
    __syncthreads();
    if (t == 0) s_last = atomicAdd(done + r, 1u) == (unsigned)(nchunks - 1);
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (t < kHcOut + kHcGram) {                       // 34 threads, each sums one column over the chunks in chunk order
        float a = 0.f;
        for (int c0 = 0; c0 < nchunks; c0 += 8) {
            float v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) v[u] = c0 + u < nchunks ? __ldcg(part + ((size_t)r * nchunks + c0 + u) * kHcPart2 + t) : 0.f;
#pragma unroll
            for (int u = 0; u < 8; ++u) a += v[u];
        }
        mix[t] = a;
    }
    __syncthreads();
    if (t < 32) {
        // sum of squares of the residual streams = trace of the Gram matrix (diagonal entries 0, 4, 7, 9 for n = 4)
        float tr = 0.f;
        { int e = 0; for (int j = 0; j < kHcMax; ++j) for (int k = j; k < kHcMax; ++k, ++e) if (k == j && j < n) tr += mix[kHcOut + e]; }
        const float inv = rsqrtf(tr / (float)(n * hidden) + rms_eps);
        float cm = 0.f;
        const int i = (t & 15) >> 2, j = t & 3;
        const bool valid = t < 16 && i < n && j < n;
        {
            float v = valid ? mix[2 * n + i * n + j] * inv * hc_scale[2] + hc_base[2 * n + i * n + j] : -INFINITY;
            float mx = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            float e = valid ? expf(v - mx) : 0.f;
            float sm = e + __shfl_xor_sync(0xffffffffu, e, 1);
            sm += __shfl_xor_sync(0xffffffffu, sm, 2);
            cm = valid ? e / sm + hc_eps : 0.f;
            float cs = cm + __shfl_xor_sync(0xffffffffu, cm, 4);
            cs += __shfl_xor_sync(0xffffffffu, cs, 8);
            cm = valid ? cm / (cs + hc_eps) : 0.f;
            for (int it = 1; it < iters; ++it) {
                float rs = cm + __shfl_xor_sync(0xffffffffu, cm, 1);
                rs += __shfl_xor_sync(0xffffffffu, rs, 2);
                cm = valid ? cm / (rs + hc_eps) : 0.f;
                cs = cm + __shfl_xor_sync(0xffffffffu, cm, 4);
                cs += __shfl_xor_sync(0xffffffffu, cs, 8);
                cm = valid ? cm / (cs + hc_eps) : 0.f;
            }
        }
        if (valid) comb[(r * n + i) * n + j] = cm;
        // pre gates on lanes 16..19, post gates on lanes 20..23
        float pre_v = 0.f;
        if (t >= 16 && t < 16 + kHcMax && t - 16 < n) pre_v = sigmoidf_(mix[t - 16] * inv * hc_scale[0] + hc_base[t - 16]) + hc_eps;
        if (t >= 20 && t < 20 + kHcMax && t - 20 < n) post[r * n + (t - 20)] = sigmoidf_(mix[n + t - 20] * inv * hc_scale[1] + hc_base[n + t - 20]) * post_mult;
        float pj[kHcMax];
#pragma unroll
        for (int q = 0; q < kHcMax; ++q) pj[q] = __shfl_sync(0xffffffffu, pre_v, 16 + q);
        if (t == 0) {
            float quad = 0.f;
            int e = 0;
            for (int a = 0; a < kHcMax; ++a)
                for (int b = a; b < kHcMax; ++b, ++e) quad += (a == b ? 1.f : 2.f) * pj[a] * pj[b] * mix[kHcOut + e];
            float* px = prex + (size_t)r * 8;
#pragma unroll
            for (int q = 0; q < kHcMax; ++q) px[q] = pj[q];
            px[4] = rsqrtf(fmaxf(quad, 0.f) / (float)hidden + rms_eps);
            done[r] = 0;
        }
    }
}

__global__ void __launch_bounds__(256) mhc_contract_kernel(bf16* __restrict__ out, const float* __restrict__ residual, const float* __restrict__ prex,
                                                           const float* __restrict__ norm_w, int hidden, int n) {
    const int r = blockIdx.x;
    const int h = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    float4 w4 = make_float4(0, 0, 0, 0);
    if (h < hidden) w4 = *reinterpret_cast<const float4*>(norm_w + h);
    pdl_wait();
    pdl_launch_dependents();
    if (h >= hidden) return;
    const float* px = prex + (size_t)r * 8;
    const float* rp = residual + (size_t)r * n * hidden + h;
    float4 a = make_float4(0, 0, 0, 0), v[kHcMax];
#pragma unroll
    for (int j = 0; j < kHcMax; ++j) v[j] = j < n ? *reinterpret_cast<const float4*>(rp + (size_t)j * hidden) : make_float4(0, 0, 0, 0);
#pragma unroll
    for (int j = 0; j < kHcMax; ++j) {
        const float p = j < n ? px[j] : 0.f;
        a.x = fmaf(p, v[j].x, a.x); a.y = fmaf(p, v[j].y, a.y); a.z = fmaf(p, v[j].z, a.z); a.w = fmaf(p, v[j].w, a.w);
    }
    const float inv = px[4];
    bf162 o0 = __floats2bfloat162_rn(a.x * inv * w4.x, a.y * inv * w4.y), o1 = __floats2bfloat162_rn(a.z * inv * w4.z, a.w * inv * w4.w);
    uint2 pk;
    pk.x = *reinterpret_cast<uint32_t*>(&o0); pk.y = *reinterpret_cast<uint32_t*>(&o1);
    *reinterpret_cast<uint2*>(out + (size_t)r * hidden + h) = pk;
}

// Last layer: out = RMSNorm(mean_j(post[j]*x + sum_i comb[i][j]*residual[i])) * w.
__global__ void mhc_contract_norm_kernel(bf16* __restrict__ out, const float* __restrict__ residual, const float* __restrict__ x,
                                         const float* __restrict__ post, const float* __restrict__ comb,
                                         const float* __restrict__ norm_w, int hidden, int n, float rms_eps, PeerComm comm) {
    __shared__ float red[33];
    extern __shared__ float row[];
    const int r = blockIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    unsigned epoch = 0;
    if (comm.nranks) {
        epoch = *comm.epoch;
        if (comm.xchg) {
            for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
                const float v = x[(size_t)r * hidden + h];
                if (comm.xchg == 2) comm_ll_put<1>(comm, epoch, (size_t)r * hidden + h, &v);
                else comm_xchg_put<1>(comm, epoch, (size_t)r * hidden + h, &v);
            }
            if (comm.xchg != 2) comm_xchg_sync(comm, epoch, r);
        } else {
            comm_wait(comm, epoch);
        }
    }
    const float* rp = residual + (size_t)r * n * hidden;
    float pm = 0.f, cw[kHcMax];
    for (int j = 0; j < n; ++j) pm += post[r * n + j];
    for (int i = 0; i < n; ++i) {
        float s = 0.f;
        for (int j = 0; j < n; ++j) s += comb[(r * n + i) * n + j];
        cw[i] = s;
    }
    float ss = 0.f;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
        float xs_;
        if (comm.nranks && comm.xchg == 2) { const float own = x[(size_t)r * hidden + h]; comm_ll_get<1>(comm, epoch, (size_t)r * hidden + h, &own, &xs_); }
        else xs_ = comm.nranks ? (comm.xchg ? comm_xchg_get(comm, epoch, (size_t)r * hidden + h, x[(size_t)r * hidden + h])
                                            : comm_reduce(comm, epoch, (size_t)r * hidden + h))
                               : x[(size_t)r * hidden + h];
        float a = pm * xs_;
        for (int i = 0; i < n; ++i) a += cw[i] * rp[(size_t)i * hidden + h];
        a /= (float)n;
        row[h] = a;
        ss += a * a;
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)hidden + rms_eps);
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) out[(size_t)r * hidden + h] = __float2bfloat16(row[h] * inv * norm_w[h]);
    pdl_launch_dependents();
}


// Producer half of the in-kernel all-reduce for partials that a kernel without a fused epilogue has already written to
// local memory: stores x[m][n] (fp32, row stride ld) into slot[this rank] of every rank's receive buffer and publishes
// the epoch.  The consumer (add_rmsnorm / mHC kernels with `comm`) sums the slots in rank order.
__global__ void __launch_bounds__(256) comm_push_rows_kernel(const float* __restrict__ x, int ld, int N, long long total, PeerComm c) {
    pdl_wait();
    pdl_launch_dependents();
    const unsigned next_epoch = *c.epoch + 1u;
    if (c.xchg) {          // the consuming kernel exchanges the (already local) partial itself
        if ((blockIdx.x | threadIdx.x) == 0) *c.epoch = next_epoch;
        return;
    }
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long m = i / N;
        comm_push(c, next_epoch, (size_t)i, x[m * ld + (i - m * N)]);
    }
    comm_signal(c, next_epoch, gridDim.x);
    pdl_launch_dependents();
}
}  // namespace lsb
using namespace lsb;

static PeerComm comm_from_host(const void* h) {
    PeerComm c;
    c.nranks = 0;
    if (h) c = *reinterpret_cast<const PeerComm*>(h);
    return c;
}

// Push a locally computed fp32 partial [M, N] (row stride ld) as this rank's contribution to the next all-reduce epoch.
LSB_API int lsb_comm_push_rows(const void* x, int M, int N, int ld, const void* comm, void* stream) {
    if (!comm) return -1;
    const PeerComm c = comm_from_host(comm);
    const long long total = (long long)M * N;
    if (c.nranks <= 0 || total > c.cap) return -2;
    const int grid = (int)((total + 256 * 8 - 1) / (256 * 8) < 592 ? (total + 256 * 8 - 1) / (256 * 8) : 592);
    launch_pdl((comm_push_rows_kernel), grid > 0 ? grid : 1, 256, 0, (cudaStream_t)stream, (const float*)x, ld, N, total, c);
    LSB_CHECK_LAUNCH();
}

LSB_API int lsb_rmsnorm(void* out, const void* x, const void* w, int rows, int dim, int ldx, int ldo, float eps,
                        int x_is_f32, void* out_f32, void* stream) {
    cudaStream_t st = (cudaStream_t)stream;
    PeerComm nocomm;
    nocomm.nranks = 0;
    const int thr = dim >= 2048 ? 512 : 256;
    const size_t sm = (size_t)dim * 4;
    if (x_is_f32)
        launch_pdl((rmsnorm_kernel<float, false>), rows, thr, sm, st, (bf16*)out, (const float*)x, nullptr, (const float*)w, dim, ldx, ldo, 0, eps, (float*)out_f32, nocomm);
    else
        launch_pdl((rmsnorm_kernel<bf16, false>), rows, thr, sm, st, (bf16*)out, (const bf16*)x, nullptr, (const float*)w, dim, ldx, ldo, 0, eps, (float*)out_f32, nocomm);
    LSB_CHECK_LAUNCH();
}

// resid (fp32, in place) += x (fp32); out = RMSNorm(resid) * w as bf16.  With `comm`, x is the
// cross-rank sum of the partials the producing kernel pushed (fused all-reduce).
LSB_API int lsb_add_rmsnorm(void* out, void* resid, const void* x, const void* w, int rows, int dim, float eps, const void* comm,
                            void* stream) {
    const int thr = dim >= 2048 ? 512 : 256;
    launch_pdl((rmsnorm_kernel<float, true>), rows, thr, (size_t)dim * 4, (cudaStream_t)stream, (bf16*)out, (const float*)x, (float*)resid,
                                                                                   (const float*)w, dim, dim, dim, dim, eps, nullptr, comm_from_host(comm));
    LSB_CHECK_LAUNCH();
}

// residual: fp32 [rows, n, hidden] updated in place; x: fp32 [rows, hidden] sublayer output
// (or the embedding when mode == 0); post/comb: state from the previous finalize (in) and
// for the next post (out, same buffers).  part: scratch fp32 [rows, hidden/32, 25].
LSB_API int lsb_mhc_post_pre(void* out_x, void* residual, const void* x, void* post, void* comb, const void* fn,
                             const void* hc_scale, const void* hc_base, const void* norm_w, void* part, int rows,
                             int hidden, int n, int mode, int iters, float hc_eps, float rms_eps, float post_mult,
                             void* done, void* prex, const void* comm, void* stream) {
    if (hidden % kHcChunk || n > kHcMax) return -1;
    cudaStream_t st = (cudaStream_t)stream;
    const int nchunks = hidden / kHcChunk;
    if (done && prex && rows < 64 && hidden % 4 == 0) {
        // few rows: partials + finalize in one launch (last block per row), then a fully parallel contraction.
        // part must hold rows * nchunks * 36 floats, done rows zero-initialised counters, prex rows * 8 floats.
        launch_pdl((mhc_post_fused_kernel), dim3(rows, nchunks), 128, 0, st, (float*)residual, (const float*)x, (float*)post, (float*)comb,
                   (const float*)fn, (const float*)hc_scale, (const float*)hc_base, (float*)part, (unsigned*)done, (float*)prex, hidden, n, mode,
                   iters, hc_eps, rms_eps, post_mult, comm_from_host(comm));
        launch_pdl((mhc_contract_kernel), dim3(rows, (hidden / 4 + 255) / 256), 256, 0, st, (bf16*)out_x, (const float*)residual, (const float*)prex,
                   (const float*)norm_w, hidden, n);
        LSB_CHECK_LAUNCH();
    }
    const int rpb = rows >= 64 ? 16 : 1;      // many rows: amortise the mixing-matrix loads over 16 rows per block
    int nparts = nchunks;
    if (rows >= 64 && hidden % kHcWide == 0) {
        nparts = hidden / kHcWide;
        // hidden parts are the fastest grid dimension: the blocks that run together read whole rows of the residual streams (16 KB
        // runs) instead of 512-byte pieces 64 KB apart
        launch_pdl((mhc_post_partial_wide_kernel), dim3(nparts, (rows + rpb - 1) / rpb), 128, 0, st, (float*)residual, (const float*)x, (const float*)post,
                   (const float*)comb, (const float*)fn, (float*)part, hidden, n, mode, rows, rpb, comm_from_host(comm));
    } else {
        launch_pdl((mhc_post_partial_kernel), dim3((rows + rpb - 1) / rpb, nchunks), 128, 0, st, (float*)residual, (const float*)x, (const float*)post,
                   (const float*)comb, (const float*)fn, (float*)part, hidden, n, mode, rows, rpb, comm_from_host(comm));
    }
    launch_pdl((mhc_finalize_kernel), rows, 512, (size_t)hidden * 4, st, (bf16*)out_x, (const float*)residual, (const float*)part,
                                                              (const float*)hc_scale, (const float*)hc_base, (const float*)norm_w,
                                                              (float*)post, (float*)comb, hidden, n, nparts, iters, hc_eps, rms_eps, post_mult);
    LSB_CHECK_LAUNCH();
}

LSB_API int lsb_mhc_contract_norm(void* out, const void* residual, const void* x, const void* post, const void* comb,
                                  const void* norm_w, int rows, int hidden, int n, float rms_eps, const void* comm, void* stream) {
    launch_pdl((mhc_contract_norm_kernel), rows, 512, (size_t)hidden * 4, (cudaStream_t)stream, (bf16*)out, (const float*)residual, (const float*)x,
                                                                                      (const float*)post, (const float*)comb,
                                                                                      (const float*)norm_w, hidden, n, rms_eps, comm_from_host(comm));
    LSB_CHECK_LAUNCH();
}

// out[r] = cos(a[r], b[r]) over `dim` bf16 elements (0 when either vector is all zero): how much a layer changed its input.
__global__ void __launch_bounds__(256) cosine_sim_kernel(const bf16* __restrict__ a, const bf16* __restrict__ b, int dim, int lda, int ldb,
                                                         float* __restrict__ out) {
    __shared__ float red[3][33];
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x;
    float ab = 0.f, aa = 0.f, bb = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const float x = __bfloat162float(a[(size_t)r * lda + i]), y = __bfloat162float(b[(size_t)r * ldb + i]);
        ab = fmaf(x, y, ab); aa = fmaf(x, x, aa); bb = fmaf(y, y, bb);
    }
    ab = block_sum(ab, red[0]); aa = block_sum(aa, red[1]); bb = block_sum(bb, red[2]);
    if (threadIdx.x == 0) out[r] = (aa > 0.f && bb > 0.f) ? ab * rsqrtf(aa) * rsqrtf(bb) : 0.f;
}

// Cosine similarity of `rows` pairs of bf16 vectors (layer skipping: the input of a layer against the input of the next one).
// Reference: src/compute/kernels/similarity/cosine_sim.h (one pair per call, output on the device).
LSB_API int lsb_cosine_sim(const void* a, const void* b, int rows, int dim, int lda, int ldb, void* out, void* stream) {
    if (rows <= 0 || dim <= 0) return -1;
    launch_pdl((cosine_sim_kernel), rows, 256, 0, (cudaStream_t)stream, (const bf16*)a, (const bf16*)b, dim, lda, ldb, (float*)out);
    LSB_CHECK_LAUNCH();
}

namespace lsb {
// ---- norms of the residual stream, on a sublayer's output and in front of the next sublayer ----
enum { kNormRms = 0, kNormLayer = 1, kNormTanh = 2, kNormNone = 3 };    // kNormTanh: dynamic tanh, b + w tanh(alpha x), element-wise
struct NormW { const float* w; const float* b; const float* alpha; int dim; float eps; int kind; };      // b may be null
__host__ __device__ __forceinline__ bool norm_moments_needed(int kind) { return kind == kNormRms || kind == kNormLayer; }

// row[0..dim) (shared memory) -> scale and shift of its normalisation: n(x) = (x - mean) * rstd
__device__ __forceinline__ void norm_moments(const float* row, const NormW& n, float* red, float& mean, float& rstd) {
    mean = 0.f;
    rstd = 1.f;
    if (!norm_moments_needed(n.kind)) return;
    if (n.kind == kNormLayer) {
        float s = 0.f;
        for (int i = threadIdx.x; i < n.dim; i += blockDim.x) s += row[i];
        mean = block_sum(s, red) / (float)n.dim;
    }
    float v = 0.f;
    for (int i = threadIdx.x; i < n.dim; i += blockDim.x) { const float d = row[i] - mean; v = fmaf(d, d, v); }
    rstd = 1.f / sqrtf(block_sum(v, red) / (float)n.dim + n.eps);
}
// element i of the normalised row; alpha: *n.alpha (dynamic tanh)
__device__ __forceinline__ float norm_apply(float v, int i, const NormW& n, float mean, float rstd, float alpha) {
    if (n.kind == kNormNone) return v;
    const float y = n.kind == kNormTanh ? tanhf(alpha * v) : (v - mean) * rstd;
    return y * n.w[i] + (n.b ? n.b[i] : 0.f);
}
template <typename T> __device__ __forceinline__ T as_act(float v);
template <> __device__ __forceinline__ bf16 as_act<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float as_act<float>(float v) { return v; }

// The sum of a row's expert outputs, slots in order: slot s holds expert ids[s]; ids below `experts` take their row of y (none when the expert is not
// resident), the others are identity experts and take the residual stream itself.  wts null: every weight is 1.
struct MoeSum { const float* y; const float* wts; const int* ids; const int* slot_of; int S, experts, ldy; };

__device__ __forceinline__ void load_slots(const MoeSum& mo, int r, int* s_id, float* s_w) {
    if ((int)threadIdx.x < mo.S) {
        int id = mo.ids[(size_t)r * mo.S + threadIdx.x];
        if (id >= 0 && id < mo.experts && mo.slot_of[id] < 0) id = -1;
        s_id[threadIdx.x] = id;
        s_w[threadIdx.x] = mo.wts ? mo.wts[(size_t)r * mo.S + threadIdx.x] : 1.f;
    }
    __syncthreads();
}
__device__ __forceinline__ float4 sum_slots4(float4 a, const MoeSum& mo, const float* yr, const float* rr, int i, const int* s_id, const float* s_w) {
#pragma unroll 4
    for (int s = 0; s < mo.S; ++s) {
        const int id = s_id[s];
        if (id < 0) continue;
        const float4 v = *reinterpret_cast<const float4*>(id < mo.experts ? yr + (size_t)s * mo.ldy + i : rr + i);
        const float w = s_w[s];
        a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
    }
    return a;
}
__device__ __forceinline__ float sum_slots(float a, const MoeSum& mo, const float* yr, const float* rr, int i, const int* s_id, const float* s_w) {
    for (int s = 0; s < mo.S; ++s) {
        const int id = s_id[s];
        if (id >= 0) a = fmaf(s_w[s], id < mo.experts ? yr[(size_t)s * mo.ldy + i] : rr[i], a);
    }
    return a;
}

// 16 bytes of activations as fp32 and back; four of them
__device__ __forceinline__ void load_act16(const float* p, float (&v)[4]) { *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void load_act16(const bf16* p, float (&v)[8]) { unpack_bf16x8(*reinterpret_cast<const uint4*>(p), v); }
__device__ __forceinline__ void store_act4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store_act4(bf16* p, const float* v) {
    const bf162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ void store_act16(float* p, const float (&v)[4]) { store_act4(p, v); }
__device__ __forceinline__ void store_act16(bf16* p, const float (&v)[8]) {
    bf162 h[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) h[u] = __floats2bfloat162_rn(v[2 * u], v[2 * u + 1]);
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(h);
}

// Causal convolution over time on the sublayer's input h = x[r], added to it: xc = h + sum_j w[j] h_(t - taps + 1 + j).  state: a sequence slot's last
// taps - 1 inputs, oldest first.  (As part of the residual update: steps of one row per sequence.)
struct InputConv { void* xc; const float* w; float* state; const int* slot; int taps, ldw; };      // w [taps, ldw], state [slots, taps - 1, ldw]

// resid[r] += post(sub[r] + MoE sum of the row) (+ step), x[r] = pre(the new residual) in the activation type.  sub may be null.  Whole rows per block.
// PLAIN: post is an RMS or layer norm and there is no pre norm, no step and no convolution.
template <typename T, bool MOE, bool PLAIN>
__global__ void __launch_bounds__(1024) post_norm_kernel(T* __restrict__ x, int ldx, float* __restrict__ resid, int ldr, const float* __restrict__ sub, int lds,
                                                        NormW post, NormW pre, MoeSum mo, const float* __restrict__ step, InputConv ic) {
    __shared__ float red[33], s_w[32];
    __shared__ int s_id[32];
    extern __shared__ float row[];
    const int r = blockIdx.x, dim = post.dim;
    float* rr = resid + (size_t)r * ldr;
    pdl_wait();
    pdl_launch_dependents();
    const float* sr = sub ? sub + (size_t)r * lds : nullptr;
    if (MOE) {
        load_slots(mo, r, s_id, s_w);
        const float* yr = mo.y + (size_t)r * mo.S * mo.ldy;
        if (dim % 4 == 0 && mo.ldy % 4 == 0 && ldr % 4 == 0 && lds % 4 == 0) {
            for (int i = threadIdx.x * 4; i < dim; i += blockDim.x * 4)
                *reinterpret_cast<float4*>(row + i) = sum_slots4(sr ? *reinterpret_cast<const float4*>(sr + i) : make_float4(0.f, 0.f, 0.f, 0.f), mo, yr, rr, i, s_id, s_w);
        } else {
            for (int i = threadIdx.x; i < dim; i += blockDim.x) row[i] = sum_slots(sr ? sr[i] : 0.f, mo, yr, rr, i, s_id, s_w);
        }
    } else {
        for (int i = threadIdx.x; i < dim; i += blockDim.x) row[i] = sr ? sr[i] : 0.f;
    }
    __syncthreads();
    float mean, rstd;
    norm_moments(row, post, red, mean, rstd);
    const float a_post = post.alpha ? *post.alpha : 0.f, a_pre = pre.alpha ? *pre.alpha : 0.f;
    T* xr = x + (size_t)r * ldx;
    if constexpr (PLAIN) {
        for (int i = threadIdx.x; i < dim; i += blockDim.x) {
            const float v = rr[i] + ((row[i] - mean) * rstd * post.w[i] + (post.b ? post.b[i] : 0.f));
            rr[i] = v;
            xr[i] = as_act<T>(v);
        }
        return;
    }
    const bool again = norm_moments_needed(pre.kind);
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const float v = rr[i] + norm_apply(row[i], i, post, mean, rstd, a_post) + (step ? step[i] : 0.f);
        rr[i] = v;
        if (again) row[i] = v;
        else xr[i] = as_act<T>(norm_apply(v, i, pre, 0.f, 1.f, a_pre));
    }
    if (!again) return;
    __syncthreads();
    norm_moments(row, pre, red, mean, rstd);
    if (!ic.xc) {
        for (int i = threadIdx.x; i < dim; i += blockDim.x) xr[i] = as_act<T>(norm_apply(row[i], i, pre, mean, rstd, a_pre));
        return;
    }
    const int slot = ic.slot[r], K = ic.taps - 1;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const T h = as_act<T>(norm_apply(row[i], i, pre, mean, rstd, a_pre));
        const float v = (float)h;
        float a = v * ic.w[(size_t)K * ic.ldw + i];
        if (slot >= 0) {
            float* s = ic.state + (size_t)slot * K * ic.ldw + i;
            for (int j = 0; j < K; ++j) {
                a = fmaf(s[(size_t)j * ic.ldw], ic.w[(size_t)j * ic.ldw + i], a);
                s[(size_t)j * ic.ldw] = j + 1 < K ? s[(size_t)(j + 1) * ic.ldw] : v;
            }
        }
        xr[i] = h;
        reinterpret_cast<T*>(ic.xc)[(size_t)r * ldx + i] = as_act<T>(v + a);
    }
}

// x = norm(resid), xc = x + conv(x) behind the residual update of steps with one row per sequence, for norms of the sum (RMS, layer norm) behind a plain update:
// a row per block, four columns per thread kept in registers; everything that the previous kernel does not write is fetched in front of the dependency wait.
template <typename T, bool MOE, int TAPS>
__global__ void __launch_bounds__(1024) norm_conv_kernel(T* __restrict__ x, int ldx, float* __restrict__ resid, int ldr, const float* __restrict__ sub, int lds, NormW pre,
                                                         MoeSum mo, const float* __restrict__ step, InputConv ic) {
    __shared__ float red[33], s_w[32];
    __shared__ int s_id[32];
    constexpr int K = TAPS - 1;
    const int r = blockIdx.x, i = threadIdx.x * 4, slot = ic.slot[r];
    const bool in = i < pre.dim;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto ld = [&](const float* p) { return p && in ? *reinterpret_cast<const float4*>(p + i) : zero; };
    float* s0 = ic.state + (size_t)max(slot, 0) * K * ic.ldw + i;
    const float4 nw = ld(pre.w), nb = ld(pre.b);
    float4 cw[TAPS], st[K ? K : 1], v = ld(step);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) cw[j] = ld(ic.w + (size_t)j * ic.ldw);
#pragma unroll
    for (int j = 0; j < K; ++j) st[j] = slot >= 0 && in ? *reinterpret_cast<const float4*>(s0 + (size_t)j * ic.ldw) : zero;
    pdl_wait();
    pdl_launch_dependents();
    if (MOE) load_slots(mo, r, s_id, s_w);
    if (in) {
        float* rr = resid + (size_t)r * ldr;
        const float4 o = *reinterpret_cast<const float4*>(rr + i);
        float4 a = ld(sub ? sub + (size_t)r * lds : nullptr);
        if (MOE) a = sum_slots4(a, mo, mo.y + (size_t)r * mo.S * mo.ldy, rr, i, s_id, s_w);
        v.x += o.x + a.x; v.y += o.y + a.y; v.z += o.z + a.z; v.w += o.w + a.w;
        *reinterpret_cast<float4*>(rr + i) = v;
    }
    if (pre.kind == kNormLayer) {
        const float mean = block_sum(v.x + v.y + v.z + v.w, red) / (float)pre.dim;
        if (in) { v.x -= mean; v.y -= mean; v.z -= mean; v.w -= mean; }
    }
    const float rstd = 1.f / sqrtf(block_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))), red) / (float)pre.dim + pre.eps);
    if (!in) return;
    const float n[4] = {v.x * rstd * nw.x + nb.x, v.y * rstd * nw.y + nb.y, v.z * rstd * nw.z + nb.z, v.w * rstd * nw.w + nb.w};
    float h[4], c[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        h[u] = (float)as_act<T>(n[u]);
        float a = h[u] * reinterpret_cast<const float*>(&cw[K])[u];
#pragma unroll
        for (int j = 0; j < K; ++j) a = fmaf(reinterpret_cast<const float*>(&st[j])[u], reinterpret_cast<const float*>(&cw[j])[u], a);
        c[u] = h[u] + a;
    }
    store_act4(x + (size_t)r * ldx + i, h);
    store_act4(reinterpret_cast<T*>(ic.xc) + (size_t)r * ldx + i, c);
    if (slot >= 0) {
#pragma unroll
        for (int j = 0; j < K; ++j) *reinterpret_cast<float4*>(s0 + (size_t)j * ic.ldw) = j + 1 < K ? st[j + 1] : make_float4(h[0], h[1], h[2], h[3]);
    }
}

// The input convolution of runs of rows: xc = x + conv(x), and every sequence's state moves on.  A block takes kConvRows rows of one sequence and V columns
// per thread (16 bytes); the inputs that the convolution looks back at stay in registers (TAPS; 0: any number of taps, read again per tap).  The first block
// of a sequence alone touches its state (the rows that the others need beyond their own are read from x).
constexpr int kConvRows = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) input_conv_kernel(const T* __restrict__ x, int ldx, InputConv ic, const int* __restrict__ seq_row0, const int* __restrict__ seq_nrows,
                                                         const int* __restrict__ seq_slot, int nseq, int dim) {
    constexpr int V = 16 / (int)sizeof(T);
    const int i = (blockIdx.x * 128 + threadIdx.x) * V, K = TAPS ? TAPS - 1 : ic.taps - 1;
    const float* w = ic.w + i;
    float cw[TAPS ? TAPS : 1][V];
    if (TAPS && i < dim) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int u = 0; u < V; u += 4) *reinterpret_cast<float4*>(&cw[j][u]) = *reinterpret_cast<const float4*>(w + (size_t)j * ic.ldw + u);
    }
    pdl_wait();
    pdl_launch_dependents();
    int tile = blockIdx.y, s = 0, n = 0;
    for (; s < nseq; ++s) {
        n = seq_nrows[s];
        const int nt = (n + kConvRows - 1) / kConvRows;
        if (tile < nt) break;
        tile -= nt;
    }
    if (s == nseq || i >= dim) return;
    const T* xs = x + (size_t)seq_row0[s] * ldx + i;
    T* out = reinterpret_cast<T*>(ic.xc) + (size_t)seq_row0[s] * ldx + i;
    float* st = ic.state + (size_t)seq_slot[s] * K * ic.ldw + i;
    auto load = [&](int t, float (&v)[V]) {                        // input of row t of the run; t < 0: before the run
        if (t >= 0) { load_act16(xs + (size_t)t * ldx, v); return; }
#pragma unroll
        for (int u = 0; u < V; u += 4) *reinterpret_cast<float4*>(&v[u]) = *reinterpret_cast<const float4*>(st + (size_t)(K + t) * ic.ldw + u);
    };
    const int r0 = tile * kConvRows, r1 = min(n, r0 + kConvRows);
    if constexpr (TAPS > 0) {
        float b[TAPS][V];                                          // the last inputs, row r in b[(r - r0 + K) % TAPS]
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) load(r0 - K + j, b[j]);
#pragma unroll
        for (int rr = 0; rr < kConvRows; ++rr) {
            if (r0 + rr >= r1) break;
            load(r0 + rr, b[(rr + TAPS - 1) % TAPS]);
            float a[V];
#pragma unroll
            for (int u = 0; u < V; ++u) {
                const float h = b[(rr + TAPS - 1) % TAPS][u];
                a[u] = h * cw[TAPS - 1][u];
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) a[u] = fmaf(b[(rr + j) % TAPS][u], cw[j][u], a[u]);
                a[u] += h;
            }
            store_act16(out + (size_t)(r0 + rr) * ldx, a);
        }
    } else {
        for (int r = r0; r < r1; ++r) {
            float h[V], a[V], b[V];
            load(r, h);
#pragma unroll
            for (int u = 0; u < V; ++u) a[u] = h[u] * w[(size_t)K * ic.ldw + u];
            for (int j = 0; j < K; ++j) {
                load(r - K + j, b);
#pragma unroll
                for (int u = 0; u < V; ++u) a[u] = fmaf(b[u], w[(size_t)j * ic.ldw + u], a[u]);
            }
#pragma unroll
            for (int u = 0; u < V; ++u) a[u] += h[u];
            store_act16(out + (size_t)r * ldx, a);
        }
    }
    // the block that reads the old state is the one that replaces it; oldest first, so that entries are read before they are overwritten.  (Tiles behind the
    // first reach back into rows of the run only: it has at least K rows in front of them.)
    if (tile == 0)
        for (int j = 0; j < K; ++j) {
            float v[V];
            load(n - K + j, v);
#pragma unroll
            for (int u = 0; u < V; u += 4) *reinterpret_cast<float4*>(st + (size_t)j * ic.ldw + u) = *reinterpret_cast<const float4*>(&v[u]);
        }
}

// The same with element-wise norms on both sides: columns spread over blocks, four per thread, nothing exchanged.
template <typename T, bool MOE>
__global__ void __launch_bounds__(128) post_norm_wide_kernel(T* __restrict__ x, int ldx, float* __restrict__ resid, int ldr, const float* __restrict__ sub, int lds,
                                                            NormW post, NormW pre, MoeSum mo) {
    __shared__ float s_w[32];
    __shared__ int s_id[32];
    const int r = blockIdx.y, i = (blockIdx.x * 128 + threadIdx.x) * 4;
    // the norms' vectors do not depend on the previous kernel: have them here before the dependency wait
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f), zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool in = i < post.dim;
    auto vec = [&](const float* v, float4 other) { return v && in ? *reinterpret_cast<const float4*>(v + i) : other; };
    const float4 w0 = vec(post.w, one), b0 = vec(post.b, zero), w1 = vec(pre.w, one), b1 = vec(pre.b, zero);
    const float a_post = post.alpha ? *post.alpha : 0.f, a_pre = pre.alpha ? *pre.alpha : 0.f;
    pdl_wait();
    pdl_launch_dependents();
    if (MOE) load_slots(mo, r, s_id, s_w);
    if (!in) return;
    float* rr = resid + (size_t)r * ldr;
    float4 a = sub ? *reinterpret_cast<const float4*>(sub + (size_t)r * lds + i) : zero;
    const float4 x0 = *reinterpret_cast<const float4*>(rr + i);
    if (MOE) a = sum_slots4(a, mo, mo.y + (size_t)r * mo.S * mo.ldy, rr, i, s_id, s_w);
    auto ew = [](float v, int kind, float alpha, float w, float b) { return kind == kNormTanh ? fmaf(tanhf(alpha * v), w, b) : v; };
    const float4 v = make_float4(x0.x + ew(a.x, post.kind, a_post, w0.x, b0.x), x0.y + ew(a.y, post.kind, a_post, w0.y, b0.y),
                                 x0.z + ew(a.z, post.kind, a_post, w0.z, b0.z), x0.w + ew(a.w, post.kind, a_post, w0.w, b0.w));
    *reinterpret_cast<float4*>(rr + i) = v;
    T* xr = x + (size_t)r * ldx + i;
    const float y[4] = {ew(v.x, pre.kind, a_pre, w1.x, b1.x), ew(v.y, pre.kind, a_pre, w1.y, b1.y), ew(v.z, pre.kind, a_pre, w1.z, b1.z), ew(v.w, pre.kind, a_pre, w1.w, b1.w)};
    if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<bf162*>(xr) = __floats2bfloat162_rn(y[0], y[1]);
        *reinterpret_cast<bf162*>(xr + 2) = __floats2bfloat162_rn(y[2], y[3]);
    } else {
        *reinterpret_cast<float4*>(xr) = make_float4(y[0], y[1], y[2], y[3]);
    }
}

// out[j] = norm(resid[rows ? rows[j] : row0 + j])
template <typename T>
__global__ void __launch_bounds__(1024) norm_rows_kernel(T* __restrict__ out, int ldo, const float* __restrict__ resid, int ldr, const int* __restrict__ rows,
                                                        int row0, NormW n) {
    __shared__ float red[33];
    extern __shared__ float row[];
    pdl_wait();
    pdl_launch_dependents();
    const float* rr = resid + (size_t)(rows ? rows[blockIdx.x] : row0 + (int)blockIdx.x) * ldr;
    for (int i = threadIdx.x; i < n.dim; i += blockDim.x) row[i] = rr[i];
    __syncthreads();
    float mean, rstd;
    norm_moments(row, n, red, mean, rstd);
    const float alpha = n.alpha ? *n.alpha : 0.f;
    for (int i = threadIdx.x; i < n.dim; i += blockDim.x)
        out[(size_t)blockIdx.x * ldo + i] = as_act<T>(norm_apply(row[i], i, n, mean, rstd, alpha));
}
static int norm_threads(int dim, int rows) { return dim >= 2048 ? (rows <= 64 ? 1024 : 512) : (dim >= 512 ? 256 : 128); }

static int residual_update(void* x, int ldx, void* resid, int ldr, const void* sub, int lds, const NormW& post, const NormW& pre, const MoeSum& mo, int rows,
                           const float* step, const InputConv& ic, int f32, cudaStream_t st) {
    const int dim = post.dim;
    if (dim < 1 || dim > 12000 || rows < 1 || (mo.y && mo.S > 32)) return -1;
    for (const NormW* n : {&post, &pre})
        if (n->kind < 0 || n->kind > kNormNone || (n->kind != kNormNone && !n->w) || (n->kind == kNormTanh && !n->alpha)) return -1;
    if (ic.xc && (!norm_moments_needed(pre.kind) || ic.taps < 1 || !ic.w || (ic.taps > 1 && !ic.state) || !ic.slot)) return -1;
    if (ic.xc && post.kind == kNormNone && ic.taps <= 4 && dim <= 4096 && !((dim | ldx | ldr | lds | ic.ldw) & 3) && (!mo.y || mo.ldy % 4 == 0)) {
        const int threads = (dim / 4 + 31) / 32 * 32;
#define LSB_NC(T, M, N) launch_pdl((norm_conv_kernel<T, M, N>), rows, threads, 0, st, (T*)x, ldx, (float*)resid, ldr, (const float*)sub, lds, pre, mo, step, ic)
#define LSB_NM(T, M) switch (ic.taps) { case 1: LSB_NC(T, M, 1); break; case 2: LSB_NC(T, M, 2); break; case 3: LSB_NC(T, M, 3); break; default: LSB_NC(T, M, 4); }
        if (f32) { if (mo.y) { LSB_NM(float, true) } else { LSB_NM(float, false) } }
        else { if (mo.y) { LSB_NM(bf16, true) } else { LSB_NM(bf16, false) } }
#undef LSB_NM
#undef LSB_NC
        LSB_CHECK_LAUNCH();
    }
    if (!step && !norm_moments_needed(post.kind) && !norm_moments_needed(pre.kind) && dim % 4 == 0 && ldx % 4 == 0 && ldr % 4 == 0 && lds % 4 == 0 && mo.ldy % 4 == 0 && rows < 65536) {
        const dim3 grid((dim / 4 + 127) / 128, rows);
#define LSB_PW(T, M) launch_pdl((post_norm_wide_kernel<T, M>), grid, 128, 0, st, (T*)x, ldx, (float*)resid, ldr, (const float*)sub, lds, post, pre, mo)
        if (f32) { if (mo.y) LSB_PW(float, true); else LSB_PW(float, false); }
        else { if (mo.y) LSB_PW(bf16, true); else LSB_PW(bf16, false); }
#undef LSB_PW
        LSB_CHECK_LAUNCH();
    }
    const bool plain = norm_moments_needed(post.kind) && pre.kind == kNormNone && !step;
#define LSB_PN(T, M) if (plain) LSB_PM(T, M, true); else LSB_PM(T, M, false)
#define LSB_PM(T, M, P) launch_pdl((post_norm_kernel<T, M, P>), rows, norm_threads(dim, rows), (size_t)dim * 4, st, (T*)x, ldx, (float*)resid, ldr, (const float*)sub, lds, post, pre, mo, step, ic)
    if (f32) { if (mo.y) { LSB_PN(float, true); } else { LSB_PN(float, false); } }
    else { if (mo.y) { LSB_PN(bf16, true); } else { LSB_PN(bf16, false); } }
#undef LSB_PN
#undef LSB_PM
    LSB_CHECK_LAUNCH();
}
}  // namespace lsb

// Residual update with a norm on either side: resid += post(sub + sum of the row's S expert outputs), x = pre(resid).  Kinds: 0 RMS, 1 layer norm,
// 2 dynamic tanh (w, b, alpha: one number), 3 none (post: the sum as it is).  sub null: no dense part; y null: no experts; wts null: experts are
// added as they are; ids >= experts: identity experts.  step [dim] (null: none) is added to the residual stream as well.  xc (null: none): the input
// convolution of steps with one row per sequence (see InputConv); slots: per row, -1 for idle rows.
LSB_API int lsb_resid_update(void* x, int ldx, void* resid, int ldr, const void* sub, int lds, int post_kind, const void* post_w, const void* post_b,
                             const void* post_alpha, int pre_kind, const void* pre_w, const void* pre_b, const void* pre_alpha, int rows, int dim,
                             float eps, const void* y, const void* wts, const void* ids, const void* slot_of, int S, int experts, int ldy, const void* step,
                             void* xc, const void* conv_w, void* conv_state, const void* slots, int taps, int ldw, int f32, void* stream) {
    const NormW post{(const float*)post_w, (const float*)post_b, (const float*)post_alpha, dim, eps, post_kind};
    const NormW pre{(const float*)pre_w, (const float*)pre_b, (const float*)pre_alpha, dim, eps, pre_kind};
    const MoeSum mo{(const float*)y, (const float*)wts, (const int*)ids, (const int*)slot_of, S, experts, ldy};
    return residual_update(x, ldx, resid, ldr, sub, lds, post, pre, mo, rows, (const float*)step, InputConv{xc, (const float*)conv_w, (float*)conv_state, (const int*)slots, taps, ldw}, f32,
                           (cudaStream_t)stream);
}

// Input convolution of a step with runs of rows: xc = x + conv(x), rows of ldx; w [taps, ldw] fp32 (last tap: the current token), state [slots, taps - 1, ldw].
LSB_API int lsb_input_conv(void* xc, const void* x, int ldx, const void* w, void* state, int taps, int ldw, const void* seq_row0, const void* seq_nrows, const void* seq_slot,
                           int nseq, int rows, int dim, int f32, void* stream) {
    if (rows < 1 || nseq < 1 || taps < 1 || taps - 1 > kConvRows || (taps > 1 && !state) || dim % 8 || ldx % 8 || ldw % 4 || ldw < dim) return -1;
    const InputConv ic{xc, (const float*)w, (float*)state, nullptr, taps, ldw};
    const int v = f32 ? 4 : 8;
    const dim3 grid((dim / v + 127) / 128, rows / kConvRows + nseq);
    cudaStream_t st = (cudaStream_t)stream;
#define LSB_IT(T, N) launch_pdl((input_conv_kernel<T, N>), grid, 128, 0, st, (const T*)x, ldx, ic, (const int*)seq_row0, (const int*)seq_nrows, (const int*)seq_slot, nseq, dim)
#define LSB_IC(T) switch (taps) { case 2: LSB_IT(T, 2); break; case 3: LSB_IT(T, 3); break; case 4: LSB_IT(T, 4); break; default: LSB_IT(T, 0); }
    if (f32) { LSB_IC(float) } else { LSB_IC(bf16) }
#undef LSB_IC
#undef LSB_IT
    LSB_CHECK_LAUNCH();
}

// out[j] = norm(resid[row]); kind as above.
LSB_API int lsb_norm_rows(void* out, int ldo, const void* resid, int ldr, const void* row_idx, int row0, const void* w, const void* b, const void* alpha,
                          int rows, int dim, float eps, int kind, int f32, void* stream) {
    if (dim < 1 || dim > 12000 || kind < 0 || kind > kNormTanh || (kind == kNormTanh && !alpha)) return -1;
    NormW n{(const float*)w, (const float*)b, (const float*)alpha, dim, eps, kind};
    cudaStream_t st = (cudaStream_t)stream;
    if (f32) launch_pdl((norm_rows_kernel<float>), rows, norm_threads(dim, rows), (size_t)dim * 4, st, (float*)out, ldo, (const float*)resid, ldr, (const int*)row_idx, row0, n);
    else launch_pdl((norm_rows_kernel<bf16>), rows, norm_threads(dim, rows), (size_t)dim * 4, st, (bf16*)out, ldo, (const float*)resid, ldr, (const int*)row_idx, row0, n);
    LSB_CHECK_LAUNCH();
}

namespace lsb {
// ---- hyper-connections with static mixing: n copies of the residual stream per row ----
// x_t <- sum_s mix[s][t] x_s + out[t] mult y for all t at once, u = sum_t in[t] x_t (in null: plain sum), next input = pre(u).
// y: the sublayer's result sub; with norms (w_a) the mean of sub and sub2, each RMS-normed; plus the row's expert sum.
struct StreamMix { const float* mix; const float* out; const float* in; float mult; };
struct StreamSub { const float* a; const float* b; int ld; const float* w_a; const float* w_b; };

template <int V> __device__ __forceinline__ void ldv(const float* p, float (&v)[V]) {
    if constexpr (V == 4) { const float4 f = *reinterpret_cast<const float4*>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
    else v[0] = *p;
}
template <int V> __device__ __forceinline__ void stv(float* p, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}

// first: [rows, ldr], the streams' common start (mix, out and y are not used).  sum: [rows, ldr] takes u (or null).  x may be null.
template <typename T, int N, int V>
__global__ void __launch_bounds__(1024) stream_update_kernel(T* __restrict__ x, int ldx, float* __restrict__ streams, int ldr, int n, const float* __restrict__ first,
                                                            float* __restrict__ sum, StreamSub sub, StreamMix hc, NormW pre, MoeSum mo) {
    constexpr int NS = N ? N : 8;
    __shared__ float red[33], s_w[32], s_mix[NS * NS], s_out[NS], s_in[NS];
    __shared__ int s_id[32];
    extern __shared__ float row[];
    const int r = blockIdx.x, dim = pre.dim, cnt = N ? N : n, t0 = threadIdx.x * V, dt = blockDim.x * V;
    if ((int)threadIdx.x < cnt * cnt && !first) s_mix[threadIdx.x / cnt * NS + threadIdx.x % cnt] = hc.mix[threadIdx.x];
    if ((int)threadIdx.x < cnt) { s_out[threadIdx.x] = first ? 0.f : hc.mult * hc.out[threadIdx.x]; s_in[threadIdx.x] = hc.in ? hc.in[threadIdx.x] : 1.f; }
    pdl_wait();
    pdl_launch_dependents();
    if (mo.y) load_slots(mo, r, s_id, s_w);
    __syncthreads();
    const float* pa = sub.a ? sub.a + (size_t)r * sub.ld : nullptr;
    const float* pb = sub.b ? sub.b + (size_t)r * sub.ld : nullptr;
    float ra = 1.f, rb = 1.f;
    if (sub.w_a) {
        float qa = 0.f, qb = 0.f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) { qa = fmaf(pa[i], pa[i], qa); qb = fmaf(pb[i], pb[i], qb); }
        ra = 0.5f / sqrtf(block_sum(qa, red) / (float)dim + pre.eps);
        rb = 0.5f / sqrtf(block_sum(qb, red) / (float)dim + pre.eps);
    }
    float* st = streams + (size_t)r * cnt * ldr;
    for (int i = t0; i < dim; i += dt) {
        float nx[NS][V], u[V];
        if (first) {
            float f[V];
            ldv<V>(first + (size_t)r * ldr + i, f);
#pragma unroll
            for (int t = 0; t < NS; ++t)
#pragma unroll
                for (int v = 0; v < V; ++v) nx[t][v] = f[v];
        } else {
            float y[V], o[V];
#pragma unroll
            for (int v = 0; v < V; ++v) y[v] = 0.f;
            if (pa) ldv<V>(pa + i, y);
            if (sub.w_a) {
                float w[V];
                ldv<V>(sub.w_a + i, w);
#pragma unroll
                for (int v = 0; v < V; ++v) y[v] = y[v] * ra * w[v];
                ldv<V>(pb + i, o);
                ldv<V>(sub.w_b + i, w);
#pragma unroll
                for (int v = 0; v < V; ++v) y[v] = fmaf(o[v] * rb, w[v], y[v]);
            }
            if (mo.y) {
                const float* yr = mo.y + (size_t)r * mo.S * mo.ldy + i;
#pragma unroll 4
                for (int s = 0; s < mo.S; ++s) {
                    if (s_id[s] < 0) continue;
                    ldv<V>(yr + (size_t)s * mo.ldy, o);
#pragma unroll
                    for (int v = 0; v < V; ++v) y[v] = fmaf(s_w[s], o[v], y[v]);
                }
            }
#pragma unroll
            for (int t = 0; t < NS; ++t)
#pragma unroll
                for (int v = 0; v < V; ++v) nx[t][v] = t < cnt ? s_out[t] * y[v] : 0.f;
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                if (s >= cnt) continue;
                ldv<V>(st + (size_t)s * ldr + i, o);
#pragma unroll
                for (int t = 0; t < NS; ++t)
#pragma unroll
                    for (int v = 0; v < V; ++v) nx[t][v] = t < cnt ? fmaf(s_mix[s * NS + t], o[v], nx[t][v]) : 0.f;
            }
        }
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = 0.f;
#pragma unroll
        for (int t = 0; t < NS; ++t) {
            if (t >= cnt) continue;
            stv<V>(st + (size_t)t * ldr + i, nx[t]);
#pragma unroll
            for (int v = 0; v < V; ++v) u[v] = fmaf(s_in[t], nx[t][v], u[v]);
        }
        if (sum) stv<V>(sum + (size_t)r * ldr + i, u);
        stv<V>(row + i, u);
    }
    if (!x) return;
    __syncthreads();
    float mean, rstd;
    norm_moments(row, pre, red, mean, rstd);
    const float alpha = pre.alpha ? *pre.alpha : 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) x[(size_t)r * ldx + i] = as_act<T>(norm_apply(row[i], i, pre, mean, rstd, alpha));
}

template <typename T, int V>
static void launch_streams(T* x, int ldx, float* streams, int ldr, int n, const float* first, float* sum, const StreamSub& sub, const StreamMix& hc, const NormW& pre,
                           const MoeSum& mo, int rows, cudaStream_t st) {
    const int dim = pre.dim, thr = norm_threads(dim, rows);
#define LSB_SU(N) LSB_SUV(N, V)
#define LSB_SUV(N, VV) launch_pdl((stream_update_kernel<T, N, VV>), rows, thr, (size_t)(dim + 3) / 4 * 16, st, x, ldx, streams, ldr, n, first, sum, sub, hc, pre, mo)
    switch (n) { case 1: LSB_SU(1); break; case 2: LSB_SU(2); break; case 3: LSB_SU(3); break; case 4: LSB_SU(4); break; default: LSB_SUV(0, 1); }
#undef LSB_SU
#undef LSB_SUV
}
}  // namespace lsb

// One step of the hyper-connections (see StreamMix): streams fp32 [rows, n, ldr].  `first` non-null starts them.  sub2 / w_a / w_b: the two results of mixers
// side by side and their norms' weights; y .. ldy: the expert sum as in lsb_resid_update (wts null: as they are).  x null: no norm behind it.
LSB_API int lsb_stream_update(void* x, int ldx, void* streams, int ldr, int n, const void* first, void* sum, const void* sub, const void* sub2, int lds,
                              const void* w_a, const void* w_b, const void* mix, const void* out, float mult, const void* in_next, int pre_kind,
                              const void* pre_w, const void* pre_b, const void* pre_alpha, int rows, int dim, float eps, const void* y, const void* wts,
                              const void* ids, const void* slot_of, int S, int experts, int ldy, int f32, void* stream) {
    if (rows < 1 || dim < 1 || dim > 12000 || n < 1 || n > 8 || (y && S > 32) || (!first && (!mix || !out)) || (w_a && (!sub || !sub2 || !w_b))) return -1;
    if (pre_kind < 0 || pre_kind > kNormNone || (pre_kind != kNormNone && !pre_w) || (pre_kind == kNormTanh && !pre_alpha)) return -1;
    const NormW pre{(const float*)pre_w, (const float*)pre_b, (const float*)pre_alpha, dim, eps, pre_kind};
    const MoeSum mo{(const float*)y, (const float*)wts, (const int*)ids, (const int*)slot_of, S, experts, ldy};
    const StreamMix hc{(const float*)mix, (const float*)out, (const float*)in_next, mult};
    const StreamSub sb{(const float*)sub, (const float*)sub2, lds, (const float*)w_a, (const float*)w_b};
    cudaStream_t st = (cudaStream_t)stream;
    const bool vec = dim % 4 == 0 && ldr % 4 == 0 && lds % 4 == 0 && ldy % 4 == 0;
#define LSB_SL(T, V) launch_streams<T, V>((T*)x, ldx, (float*)streams, ldr, n, (const float*)first, (float*)sum, sb, hc, pre, mo, rows, st)
    if (f32) { if (vec) LSB_SL(float, 4); else LSB_SL(float, 1); }
    else { if (vec) LSB_SL(bf16, 4); else LSB_SL(bf16, 1); }
#undef LSB_SL
    LSB_CHECK_LAUNCH();
}

LSB_API int lsb_trace_set_norm(void* buf) { return lsb_trace_install(buf); }
