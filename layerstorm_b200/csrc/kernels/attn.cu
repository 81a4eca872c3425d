// Grouped-query softmax attention over the paged cache, with an optional sliding window or chunked mask, a per-head linear or learned distance
// bias, query / key norms over the whole projection or per head, rotary positions, value mixing across layers and an output gate per channel
// or head - every one of them a parameter.
//
//   q = RMSNorm_all(W_q h), k = RMSNorm_all(W_k h)        one norm over all rows of the projection (w = null: no norm)
//   v = (1 - lambda) W_v h + lambda v_first                (mix = 2), v_first = the values of the first mixing layer (mix = 1 stores them)
//   or per head: q, k = rot(RMSNorm_head(W h + b))         norm with or without a weight, "rotate half" over the leading channels
//   s_ij = scale q_i . k_j - slope_h (i - j) + bias_h[i - j],  0 <= i - j < window (window 0: the whole prefix), i and j in one chunk;
//   o_i = softmax_j(s_ij) v_j
//   out = o * sigmoid(gate)                                (gate offset < 0: none)
//   a sink adds exp(sink_h) to the softmax's denominator; a temperature per head rides on the queries
//   differential form: two maps per head over the same values, o = rms(o_1 - lambda o_2) (1 - diff) per head
//
// Cache row of a token: [G * dkp keys | G / maps * dvp values], head widths padded with zeros to dkp / dvp.  With several maps a "head" of the
// attention kernels is one map of a query head; they are ordered [value head, map, head of the group].
//   attn_prep      norms, value mixing, append to the cache;  attn_head_prep: biases, per-head norms, rotation, temperatures, append
//   attn_decode    few rows: one block per (row, kv head, split of the visible keys); the heads of a group are the rows of mma.sync tiles, each
//                  warp walks its own 16-key tiles; attn_combine merges the splits
//   attn_prefill   runs of rows: 128 (token, head) rows of a sequence per block against 32-key tiles shared by eight warps
//   attn_diff      difference of the two maps' results and its norm, merging the few-row form's splits
//   attn_exact     fp32 cache and activations (and bf16 caches whose head widths the tensor-core kernels do not cover): CUDA cores
// Scores, weights and the output sum are fp32; the tensor-core kernels split the weights into a bf16 (hi | lo) pair for the value product.
#include "attn_core.cuh"

namespace lsb {

// ------------------------------------------------------------------------------------------------ projection -> q, cache row
template <typename T, int NT>
__global__ void __launch_bounds__(NT) attn_prep_kernel(const float* __restrict__ proj, int ldp, int off_q, int off_k, int off_v, const float* __restrict__ wq,
                                                        const float* __restrict__ wk, float eps, float* __restrict__ vfirst, int mix,
                                                        const float* __restrict__ lambda, T* __restrict__ q_out, T* __restrict__ cache,
                                                        const int* __restrict__ block_table, int max_pages, const int* __restrict__ row_seq,
                                                        const int* __restrict__ row_pos, int H, int G, int dk, int dv, int dkp, int dvp, int page) {
    __shared__ float red[2][32];
    constexpr int nt = NT;
    const int r = blockIdx.x, t = threadIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    const int seq = row_seq[r], pos = row_pos[r];
    if (seq < 0) return;
    const float* pr = proj + (size_t)r * ldp;
    T* row = cache + ((size_t)block_table[(size_t)seq * max_pages + pos / page] * page + pos % page) * ((size_t)G * (dkp + dvp));
    float qr = 1.f, kr = 1.f;
    if (wq) {
        float a = 0.f, b = 0.f;
#pragma unroll 4
        for (int i = t; i < H * dk; i += nt) { const float x = pr[off_q + i]; a = fmaf(x, x, a); }
#pragma unroll 4
        for (int i = t; i < G * dk; i += nt) { const float x = pr[off_k + i]; b = fmaf(x, x, b); }
        a = warp_sum(a); b = warp_sum(b);
        if ((t & 31) == 0) { red[0][t >> 5] = a; red[1][t >> 5] = b; }
        __syncthreads();
        a = (t & 31) < NT / 32 ? red[0][t & 31] : 0.f;            // every warp adds the warps' partials on its own
        b = (t & 31) < NT / 32 ? red[1][t & 31] : 0.f;
        qr = 1.f / sqrtf(warp_sum(a) / (float)(H * dk) + eps);
        kr = 1.f / sqrtf(warp_sum(b) / (float)(G * dk) + eps);
    }
    for (int i = t; i < H * dkp; i += nt) {
        const int h = i / dkp, c = i - h * dkp, s = h * dk + c;
        q_out[(size_t)r * H * dkp + i] = to_act<T>(c < dk ? pr[off_q + s] * qr * (wq ? wq[s] : 1.f) : 0.f);
    }
    for (int i = t; i < G * dkp; i += nt) {
        const int g = i / dkp, c = i - g * dkp, s = g * dk + c;
        row[i] = to_act<T>(c < dk ? pr[off_k + s] * kr * (wk ? wk[s] : 1.f) : 0.f);
    }
    const float lam = mix == 2 ? *lambda : 0.f;
    for (int i = t; i < G * dvp; i += nt) {
        const int g = i / dvp, c = i - g * dvp, s = g * dv + c;
        float v = 0.f;
        if (c < dv) {
            v = pr[off_v + s];
            if (mix == 1) vfirst[(size_t)r * G * dv + s] = v;
            if (mix == 2) v = (1.f - lam) * v + lam * vfirst[(size_t)r * G * dv + s];
        }
        row[G * dkp + i] = to_act<T>(v);
    }
}

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store4(bf16* p, float a, float b, float c, float d) {
    const bf162 u = __floats2bfloat162_rn(a, b), v = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&u), *reinterpret_cast<const uint32_t*>(&v));
}

// One block per row, one warp per head: q and k = rot(norm(proj + bias)), v = proj + bias.  norm 0 none, 1 without a weight, 2 with wq / wk [dk].
// Rotation of the leading `rot` channels: channel c with c + rot / 2, or (pairs) 2 i with 2 i + 1.  temp [H]: factor on a head's queries.  maps > 1: H
// and G count maps, which the projection holds as [head, map]; queries are stored as [value head, map, head of the group].
template <typename T, int NT>
__global__ void __launch_bounds__(NT) attn_head_prep_kernel(const float* __restrict__ proj, int ldp, int off_q, int off_k, int off_v, const float* __restrict__ bq,
                                                             const float* __restrict__ bk, const float* __restrict__ bv, int norm, const float* __restrict__ wq,
                                                             const float* __restrict__ wk, float eps, int rot, int pairs, const double* __restrict__ inv_freq,
                                                             const float* __restrict__ temp, int maps,
                                                             T* __restrict__ q_out, T* __restrict__ cache, const int* __restrict__ block_table, int max_pages,
                                                             const int* __restrict__ row_seq, const int* __restrict__ row_pos, int H, int G, int dk, int dv,
                                                             int dkp, int dvp, int page) {
    extern __shared__ float s_cs[];                                // [rot / 2] cosines | [rot / 2] sines
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = rot / 2;
    pdl_wait();
    pdl_launch_dependents();
    const int seq = row_seq[r], pos = row_pos[r];
    if (seq < 0) return;
    for (int i = threadIdx.x; i < half; i += NT) rotary_angle(pos, inv_freq[i], s_cs[half + i], s_cs[i]);
    __syncthreads();
    const float* pr = proj + (size_t)r * ldp;
    const int Gv = G / maps, hg = H / G;
    const bool vec = !norm && !bq && !bk && !((dk | dv | ldp | off_q | off_k | off_v | rot / 2) & 3);
    T* row = cache + ((size_t)block_table[(size_t)seq * max_pages + pos / page] * page + pos % page) * ((size_t)G * dkp + (size_t)Gv * dvp);
    for (int j = warp; j < H + G + Gv; j += NT / 32) {
        if (j >= H + G) {
            const int g = j - H - G;
            if (vec && !bv) {
                for (int c = lane * 4; c < dvp; c += 128) {
                    float v[4] = {0.f, 0.f, 0.f, 0.f};
                    if (c < dv) load4(pr + off_v + g * dv + c, v);
                    store4(row + G * dkp + g * dvp + c, v[0], v[1], v[2], v[3]);
                }
                continue;
            }
            for (int c = lane; c < dvp; c += 32)
                row[G * dkp + g * dvp + c] = to_act<T>(c < dv ? pr[off_v + g * dv + c] + (bv ? bv[g * dv + c] : 0.f) : 0.f);
            continue;
        }
        const bool isq = j < H;
        const int h = isq ? j : j - H;
        const float* x = pr + (isq ? off_q : off_k) + (size_t)h * dk;
        const float* b = isq ? bq : bk;
        const float* w = isq ? wq : wk;
        if (b) b += (size_t)h * dk;
        float rs = 1.f;
        if (norm) {
            float a = 0.f;
#pragma unroll 4
            for (int c = lane; c < dk; c += 32) { const float v = x[c] + (b ? b[c] : 0.f); a = fmaf(v, v, a); }
            rs = 1.f / sqrtf(warp_sum(a) / (float)dk + eps);
        }
        auto at = [&](int c) { return (x[c] + (b ? b[c] : 0.f)) * rs * (norm == 2 ? w[c] : 1.f); };
        const int hq = h / maps, at_q = maps > 1 ? (hq / hg * maps + h % maps) * hg + hq % hg : h;
        T* d = isq ? q_out + ((size_t)r * H + at_q) * dkp : row + (size_t)h * dkp;
        const float f = isq && temp ? temp[hq] : 1.f;
        if (vec) {                                                 // plain rotation, four channels a lane
            for (int c = lane * 4; c < dkp; c += 128) {
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                if (c < dk) {
                    load4(x + c, v);
                    if (c < rot && pairs) {
#pragma unroll
                        for (int u = 0; u < 4; u += 2) {
                            const float cs = s_cs[(c + u) >> 1], sn = s_cs[half + ((c + u) >> 1)], a = v[u], b2 = v[u + 1];
                            v[u] = a * cs - b2 * sn; v[u + 1] = b2 * cs + a * sn;
                        }
                    } else if (c < rot) {
                        float o[4];
                        const int k = c < half ? c : c - half;
                        load4(x + (c < half ? c + half : k), o);
#pragma unroll
                        for (int u = 0; u < 4; ++u) v[u] = v[u] * s_cs[k + u] + (c < half ? -o[u] : o[u]) * s_cs[half + k + u];
                    }
                }
                store4(d + c, v[0] * f, v[1] * f, v[2] * f, v[3] * f);
            }
            continue;
        }
#pragma unroll 4
        for (int c = lane; c < dkp; c += 32) {
            float v = 0.f;
            if (c < dk) {
                v = at(c);
                if (pairs) { if (c < rot) v = v * s_cs[c >> 1] + at(c ^ 1) * (c & 1 ? s_cs[half + (c >> 1)] : -s_cs[half + (c >> 1)]); }
                else if (c < half) v = v * s_cs[c] - at(c + half) * s_cs[half + c];
                else if (c < rot) v = v * s_cs[c - half] + at(c - half) * s_cs[c];
            }
            d[c] = to_act<T>(v * f);
        }
    }
}

// One warp's 16 query rows against NT 16-key tiles held in shared memory.  K: [keys][ldk], V: [keys][ldv]; row r of the warp sits at
// position pos[r / 8 half] and sees keys from low[..] on; scores are in log2 units.  m, l: running maximum and sum of the thread's two rows.
// BIAS 1: tab[row][distance] in log2 units; 2: as it is stored, distances clamped to bias_last.  MAPS 2: rows 0 - 7 attend over the keys in sk, rows 8 - 15 over
// those in sk2 (NT * 16 rows behind), both over the same values.
template <int NV, int NT, int BIAS, int MAPS = 1>
__device__ __forceinline__ void attn_tiles(const bf16* sq, int ldq, const bf16* sk, int ldk, const bf16* sv, int ldv, int dkp, int key0, int key_end,
                                           const int (&pos)[2], const int (&low)[2], float scale2, const float (&slope2)[2], const float* const (&tab)[2],
                                           int bias_last, float (&m)[2], float (&l)[2], float (&o)[NV][4]) {
    const int lane = threadIdx.x & 31;
    float s[2 * NT][4];
#pragma unroll
    for (int i = 0; i < 2 * NT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
    float s2[MAPS == 2 ? 2 * NT : 1][4];
    if constexpr (MAPS == 2) {
#pragma unroll
        for (int i = 0; i < 2 * NT; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) s2[i][j] = 0.f;
    }
    const bf16* qp = sq + (lane & 15) * ldq + (lane >> 4) * 8;
    const bf16* kp = sk + ((lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 2
    for (int k = 0; k < dkp; k += 16) {
        uint32_t a[4];
        ldsm4(a, qp + k);
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            uint32_t b[4];
            ldsm4(b, kp + t * 16 * ldk + k);
            mma_bf16(s[2 * t], a, b[0], b[1]);
            mma_bf16(s[2 * t + 1], a, b[2], b[3]);
            if constexpr (MAPS == 2) {
                ldsm4(b, kp + (NT + t) * 16 * ldk + k);
                mma_bf16(s2[2 * t], a, b[0], b[1]);
                mma_bf16(s2[2 * t + 1], a, b[2], b[3]);
            }
        }
    }
    if constexpr (MAPS == 2) {
#pragma unroll
        for (int i = 0; i < 2 * NT; ++i) { s[i][2] = s2[i][2]; s[i][3] = s2[i][3]; }
    }
    float mt[2] = {m[0], m[1]};
#pragma unroll
    for (int i = 0; i < 2 * NT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int row = j >> 1, key = key0 + (i >> 1) * 16 + (i & 1) * 8 + (lane & 3) * 2 + (j & 1), dist = pos[row] - key;
            const bool seen = dist >= 0 && key >= low[row] && key < key_end;
            if constexpr (BIAS == 0) s[i][j] = seen ? s[i][j] * scale2 - slope2[row] * (float)dist : -INFINITY;
            else if constexpr (BIAS == 1) s[i][j] = seen ? fmaf(s[i][j], scale2, tab[row][dist]) : -INFINITY;
            else s[i][j] = seen ? fmaf(s[i][j], scale2, __ldg(tab[row] + min(dist, bias_last)) * kLog2e) : -INFINITY;
            mt[row] = fmaxf(mt[row], s[i][j]);
        }
    float corr[2], base[2];
#pragma unroll
    for (int row = 0; row < 2; ++row) {
        mt[row] = fmaxf(mt[row], __shfl_xor_sync(0xffffffffu, mt[row], 1));
        mt[row] = fmaxf(mt[row], __shfl_xor_sync(0xffffffffu, mt[row], 2));
        base[row] = mt[row] == -INFINITY ? 0.f : mt[row];
        corr[row] = ex2(m[row] - base[row]);               // m = -inf: 0
        m[row] = mt[row];
        l[row] *= corr[row];
    }
    // after the first tiles the maxima rarely move; the few-row form gains by looking (163 -> 148 us for 32 sequences of 4096 keys), long tiles lose
    if (NT > 1 || __any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < NV; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
    }
    const bf16* vp = sv + ((lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8;
#pragma unroll
    for (int t = 0; t < NT; ++t) {
        float e[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int j = 0; j < 4; ++j) { e[u][j] = ex2(s[2 * t + u][j] - base[j >> 1]); l[j >> 1] += e[u][j]; }
        uint32_t hi[4], lo[4];
        split2(e[0][0], e[0][1], hi[0], lo[0]);
        split2(e[0][2], e[0][3], hi[1], lo[1]);
        split2(e[1][0], e[1][1], hi[2], lo[2]);
        split2(e[1][2], e[1][3], hi[3], lo[3]);
#pragma unroll
        for (int i = 0; i < NV; i += 2) {
            uint32_t b[4];
            ldsm4_t(b, vp + t * 16 * ldv + i * 8);
            mma_bf16(o[i], hi, b[0], b[1]);
            mma_bf16(o[i], lo, b[0], b[1]);
            mma_bf16(o[i + 1], hi, b[2], b[3]);
            mma_bf16(o[i + 1], lo, b[2], b[3]);
        }
    }
}

// ------------------------------------------------------------------------------------------------ decode
constexpr int kDecStages = 3;
// MAPS 2: both maps of up to eight heads are the rows of one tile, their keys and the values they share one stage.
template <int DVP, int BIAS, int MAPS>
__global__ void __launch_bounds__(128) attn_decode_kernel(AttnParams p) {
    constexpr int NV = DVP / 8, HB = 16 / MAPS;                    // heads of a tile
    extern __shared__ __align__(16) bf16 asm_[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = threadIdx.x;
    const int groups = p.G / MAPS, r = blockIdx.x / groups, g = blockIdx.x % groups, split = blockIdx.y, hg = p.H / p.G, h0 = blockIdx.z * HB;
    const int ldk = p.dkp + 8, ldv = DVP + 8;
    bf16* sq = asm_;                                              // [16][ldk]
    const int stage = 16 * (MAPS * ldk + ldv);
    bf16* st = sq + 16 * ldk + (size_t)warp * kDecStages * stage;
    pdl_wait();
    pdl_launch_dependents();
    const int seq = p.row_seq[r], pos = p.row_pos[r];
    if (seq < 0) return;
    const bf16* q = reinterpret_cast<const bf16*>(p.q) + (size_t)r * p.H * p.dkp;
    const int nh = min(HB, hg - h0);
    auto head = [&](int row) { return (g * MAPS + row / HB) * hg + h0 + min(row % HB, nh - 1); };
    for (int i = t; i < 16 * (p.dkp / 8); i += 128) {
        const int hh = i / (p.dkp / 8), c = i % (p.dkp / 8);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (hh % HB < nh) v = *reinterpret_cast<const uint4*>(q + (size_t)head(hh) * p.dkp + c * 8);
        *reinterpret_cast<uint4*>(sq + hh * ldk + c * 8) = v;
    }
    const int lo = attn_low(p, pos);
    const int ntile = (pos - lo + 16) / 16;                       // 16-key tiles of the visible range
    const int per = (ntile + p.NS - 1) / p.NS, t0 = split * per, t1 = min(ntile, t0 + per);
    const size_t ldc = (size_t)p.ldc;
    const bf16* cache = reinterpret_cast<const bf16*>(p.cache);
    const int kc = p.dkp / 8, vc = DVP / 8;
    auto issue = [&](int tile, int buf) {
        if (tile < t1) {
            bf16* dk_ = st + (size_t)buf * stage;
            bf16* dv_ = dk_ + MAPS * 16 * ldk;
            // two lanes per key, alternating 16-byte pieces; keys past the position are clamped (masked later)
            const int kr = lane >> 1, j = min(lo + tile * 16 + kr, pos);
            const bf16* src = cache + ((size_t)p.block_table[(size_t)seq * p.max_pages + j / p.page] * p.page + j % p.page) * ldc;
#pragma unroll
            for (int m = 0; m < MAPS; ++m)
                for (int c = lane & 1; c < kc; c += 2) cp16(dk_ + (m * 16 + kr) * ldk + c * 8, src + (size_t)(g * MAPS + m) * p.dkp + c * 8);
            for (int c = lane & 1; c < vc; c += 2) cp16(dv_ + kr * ldv + c * 8, src + (size_t)p.off_v + (size_t)(MAPS == 2 ? g : g / p.maps) * p.dvp + c * 8);
        }
        cp_commit();
    };
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    const int hr0 = head(lane >> 2), hr1 = head((lane >> 2) + 8);
    const float slope2[2] = {p.slope ? p.slope[hr0] * kLog2e : 0.f, p.slope ? p.slope[hr1] * kLog2e : 0.f};
    const int pp[2] = {pos, pos}, low[2] = {lo, lo};
    const float* const tab[2] = {BIAS ? p.bias + (size_t)hr0 * p.bias_len : nullptr, BIAS ? p.bias + (size_t)hr1 * p.bias_len : nullptr};
#pragma unroll
    for (int s = 0; s < kDecStages - 1; ++s) issue(t0 + warp + 4 * s, s);
    __syncthreads();
    int buf = 0;
    for (int tile = t0 + warp; tile < t1; tile += 4) {
        issue(tile + 4 * (kDecStages - 1), (buf + kDecStages - 1) % kDecStages);
        cp_wait<kDecStages - 1>();
        __syncwarp();
        const bf16* dk_ = st + (size_t)buf * stage;
        attn_tiles<NV, 1, BIAS ? 2 : 0, MAPS>(sq, ldk, dk_, ldk, dk_ + MAPS * 16 * ldk, ldv, p.dkp, lo + tile * 16, pos + 1, pp, low, p.scale * kLog2e, slope2, tab,
                                        p.bias_len - 1, m, l, o);
        __syncwarp();
        buf = (buf + 1) % kDecStages;
    }
    cp_wait<0>();
#pragma unroll
    for (int row = 0; row < 2; ++row) {
        l[row] += __shfl_xor_sync(0xffffffffu, l[row], 1);
        l[row] += __shfl_xor_sync(0xffffffffu, l[row], 2);
    }
    // merge the four warps through shared memory (fixed order)
    __syncthreads();
    float* so = reinterpret_cast<float*>(asm_);                   // [4][16][DVP + 2]
    constexpr int LDO = DVP + 2;
#pragma unroll
    for (int row = 0; row < 2; ++row) {
        float* d = so + ((size_t)warp * 16 + (lane >> 2) + 8 * row) * LDO;
#pragma unroll
        for (int i = 0; i < NV; ++i) { d[i * 8 + (lane & 3) * 2] = o[i][2 * row]; d[i * 8 + (lane & 3) * 2 + 1] = o[i][2 * row + 1]; }
        if ((lane & 3) == 0) { d[DVP] = m[row]; d[DVP + 1] = l[row]; }
    }
    __syncthreads();
    for (int i = t; i < MAPS * nh * p.dv; i += 128) {
        const int j = i / p.dv, c = i - j * p.dv, hh = j / nh * HB + j % nh, h = head(hh);
        float M = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) M = fmaxf(M, so[((size_t)w * 16 + hh) * LDO + DVP]);
        float L = 0.f, O = 0.f;
        if (M != -INFINITY) {
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const float* d = so + ((size_t)w * 16 + hh) * LDO;
                const float f = ex2(d[DVP] - M);
                L = fmaf(d[DVP + 1], f, L);
                O = fmaf(d[c], f, O);
            }
        }
        if (p.NS == 1) {
            O *= attn_inv_sum(p, h, M, L);
            if (p.out32) { p.out32[((size_t)r * p.H + h) * p.dvp + c] = O; continue; }
            O *= attn_out_factor(p, r, h, c);
            reinterpret_cast<bf16*>(p.out)[(size_t)r * p.ldo + (size_t)h * p.dv + c] = __float2bfloat16(O);
        } else {
            const size_t k = ((size_t)r * p.H + h) * p.NS + split;
            p.o_part[k * p.dvp + c] = O;
            if (c == 0) { p.ml_part[2 * k] = M; p.ml_part[2 * k + 1] = L; }
        }
    }
}

__global__ void __launch_bounds__(128) attn_combine_kernel(AttnParams p) {
    const int r = blockIdx.x, h = blockIdx.y;
    pdl_wait();
    pdl_launch_dependents();
    if (p.row_seq[r] < 0) return;
    const size_t k0 = ((size_t)r * p.H + h) * p.NS;
    float M = -INFINITY;
    for (int s = 0; s < p.NS; ++s) M = fmaxf(M, p.ml_part[2 * (k0 + s)]);
    float L = 0.f;
    for (int s = 0; s < p.NS; ++s) L = fmaf(p.ml_part[2 * (k0 + s) + 1], ex2(p.ml_part[2 * (k0 + s)] - M), L);
    const float inv = attn_inv_sum(p, h, M, L);
    for (int c = threadIdx.x; c < p.dv; c += 128) {
        float O = 0.f;
        for (int s = 0; s < p.NS; ++s) O = fmaf(p.o_part[(k0 + s) * p.dvp + c], ex2(p.ml_part[2 * (k0 + s)] - M), O);
        O = O * inv * attn_out_factor(p, r, h, c);
        reinterpret_cast<bf16*>(p.out)[(size_t)r * p.ldo + (size_t)h * p.dv + c] = __float2bfloat16(O);
    }
}

// Differential heads: o_1 and o_2 of head h of a row -> rms(o_1 - lambda o_2) factor.  parts [rows, 2 H, NS, dvp] in the order [value head, map, head of the
// group].  Normalised results (NS = 1): one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(128) attn_diff_kernel(T* __restrict__ out, int ldo, const float* __restrict__ parts, int H, int hg, int dv, int dvp, float lambda, float eps,
                                                        float factor, const int* __restrict__ row_seq) {
    extern __shared__ float sdiff[];                               // [4][dv]
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y * 4 + warp;
    pdl_wait();
    pdl_launch_dependents();
    if (row_seq[r] < 0 || h >= H) return;
    float* d = sdiff + warp * dv;
    const float* p1 = parts + ((size_t)r * 2 * H + h / hg * 2 * hg + h % hg) * dvp;
    const float* p2 = p1 + (size_t)hg * dvp;
    float ss = 0.f;
#pragma unroll 4
    for (int c = lane; c < dv; c += 32) {
        const float v = fmaf(-lambda, p2[c], p1[c]);
        d[c] = v;
        ss = fmaf(v, v, ss);
    }
    const float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll 4
    for (int c = lane; c < dv; c += 32) out[(size_t)r * ldo + (size_t)h * dv + c] = to_act<T>(d[c] * f);
}

// The same from split sums (maxima and sums in ml): one block per (row, head); a thread takes four channels of every ng-th split of both maps.
template <typename T>
__global__ void __launch_bounds__(256) attn_diff_merge_kernel(T* __restrict__ out, int ldo, const float* __restrict__ parts, const float* __restrict__ ml, int NS, int ng, int H,
                                                              int hg, int dv, int dvp, float lambda, float eps, float factor, const int* __restrict__ row_seq) {
    extern __shared__ __align__(16) float sdiff[];                 // [ng][4 nq]
    __shared__ float sw[2][32], red[33];
    const int r = blockIdx.x, h = blockIdx.y, t = threadIdx.x, lane = t & 31, nq = (dv + 3) / 4;
    pdl_wait();
    pdl_launch_dependents();
    if (row_seq[r] < 0) return;
    const size_t k1 = ((size_t)r * 2 * H + h / hg * 2 * hg + h % hg) * NS, k2 = k1 + (size_t)hg * NS;
    if (t < 64) {
        const size_t k = t < 32 ? k1 : k2;
        const float m = lane < NS ? ml[2 * (k + lane)] : -INFINITY, l = lane < NS ? ml[2 * (k + lane) + 1] : 0.f;
        const float M = warp_max(m), e = m == -INFINITY ? 0.f : ex2(m - M);
        sw[t >> 5][lane] = e / warp_sum(e * l) * (t < 32 ? 1.f : -lambda);
    }
    __syncthreads();
    for (int i = t; i < nq * ng; i += 256) {
        const int g = i / nq, q = i - g * nq;
        const float4* p1 = reinterpret_cast<const float4*>(parts + k1 * dvp) + q;
        const float4* p2 = reinterpret_cast<const float4*>(parts + k2 * dvp) + q;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = g; s < NS; s += ng) {
            const float4 x = p1[(size_t)s * (dvp / 4)], y = p2[(size_t)s * (dvp / 4)];
            const float u = sw[0][s], v = sw[1][s];
            a.x = fmaf(u, x.x, fmaf(v, y.x, a.x)); a.y = fmaf(u, x.y, fmaf(v, y.y, a.y)); a.z = fmaf(u, x.z, fmaf(v, y.z, a.z)); a.w = fmaf(u, x.w, fmaf(v, y.w, a.w));
        }
        reinterpret_cast<float4*>(sdiff)[i] = a;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = t; c < dv; c += 256) {
        float v = sdiff[c];
        for (int g = 1; g < ng; ++g) v += sdiff[g * 4 * nq + c];
        sdiff[c] = v;
        ss = fmaf(v, v, ss);
    }
    const float f = factor / sqrtf(block_sum(ss, red) / (float)dv + eps);
    for (int c = t; c < dv; c += 256) out[(size_t)r * ldo + (size_t)h * dv + c] = to_act<T>(sdiff[c] * f);
}

// ------------------------------------------------------------------------------------------------ prefill
constexpr int kPreKeys = 32;          // keys per tile: with 32, two 256-thread blocks fit an SM's registers (1.24 -> 0.97 ms for 2048 rows x 4096 keys x 32 heads)
// row stride of the prefill form's slices of the bias table: one slice per head and key tile, all distances a tile of tq tokens can have
__host__ __device__ constexpr int attn_bias_ld(int tq) { return (tq + kPreKeys - 1 + 31) / 32 * 32 + 8; }
template <int DVP, int BIAS>
__global__ void __launch_bounds__(256, DVP <= 128 ? 2 : 1) attn_prefill_kernel(AttnParams p, const int* __restrict__ seq_row0, const int* __restrict__ seq_nrows, int nseq,
                                                           int tq) {
    constexpr int NV = DVP / 8, kTpk = 256 / kPreKeys;             // threads per key of a tile copy
    extern __shared__ __align__(16) bf16 asm_[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = threadIdx.x, g = blockIdx.y, hg = p.H / p.G;
    const int ldk = p.dkp + 8, ldv = DVP + 8;
    bf16* sq = asm_;                                              // [128][ldk]
    bf16* skv = sq + 128 * ldk;                                   // [2][kPreKeys][ldk + ldv]
    float* sbias = reinterpret_cast<float*>(skv + 2 * kPreKeys * (ldk + ldv));     // [2][hg][attn_bias_ld]
    pdl_wait();
    pdl_launch_dependents();
    // tile -> rows [r0, r0 + n) of one sequence
    int r0 = 0, n = 0;
    for (int s = 0, base = 0; s < nseq; ++s) {
        const int ns = seq_nrows[s], nt = (ns + tq - 1) / tq;
        if ((int)blockIdx.x < base + nt) { const int k = blockIdx.x - base; r0 = seq_row0[s] + k * tq; n = min(tq, ns - k * tq); break; }
        base += nt;
    }
    if (n <= 0) return;
    const int seq = p.row_seq[r0], pos0 = p.row_pos[r0];
    if (seq < 0) return;
    const bf16* q = reinterpret_cast<const bf16*>(p.q);
    for (int i = t; i < 128 * (p.dkp / 8); i += 256) {
        const int m = i / (p.dkp / 8), c = i % (p.dkp / 8), tok = m / hg;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (tok < n) v = *reinterpret_cast<const uint4*>(q + ((size_t)(r0 + tok) * p.H + (size_t)g * hg + m % hg) * p.dkp + c * 8);
        *reinterpret_cast<uint4*>(sq + m * ldk + c * 8) = v;
    }
    const int pos_last = pos0 + n - 1;
    const int lo = max(attn_low(p, pos0) / kPreKeys * kPreKeys, p.key_base);
    const int ntile = (pos_last - lo) / kPreKeys + 1;
    const size_t ldc = (size_t)p.ldc;
    const bf16* cache = reinterpret_cast<const bf16*>(p.cache);
    const int kc = p.dkp / 8, vc = DVP / 8;
    auto issue = [&](int tile) {
        if (tile < ntile) {
            bf16* dk_ = skv + (size_t)(tile & 1) * kPreKeys * (ldk + ldv);
            bf16* dv_ = dk_ + kPreKeys * ldk;
            const int kr = t / kTpk, j = min(lo + tile * kPreKeys + kr, pos_last) - p.key_base;
            const bf16* src = cache + ((size_t)p.block_table[(size_t)seq * p.max_pages + j / p.page] * p.page + j % p.page) * ldc;
            for (int c = t % kTpk; c < kc; c += kTpk) cp16(dk_ + kr * ldk + c * 8, src + (c * 8 < p.dkh ? (size_t)g * p.dkh + c * 8 : (size_t)p.off_ks + c * 8 - p.dkh));
            for (int c = t % kTpk; c < vc; c += kTpk) cp16(dv_ + kr * ldv + c * 8, src + (size_t)p.off_v + (size_t)(g / p.maps) * p.dvp + c * 8);
            if constexpr (BIAS) {
                const int ldb = attn_bias_ld(tq), d0 = pos0 - (lo + tile * kPreKeys) - (kPreKeys - 1);       // distance of column 0
                float* sb = sbias + (tile & 1) * hg * ldb;
                for (int h = warp; h < hg; h += 8)
                    for (int c = lane; c < tq + kPreKeys - 1; c += 32)
                        sb[h * ldb + c] = __ldg(p.bias + (size_t)(g * hg + h) * p.bias_len + min(max(d0 + c, 0), p.bias_len - 1)) * kLog2e;
            }
        }
        cp_commit();
    };
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    int mr[2], pp[2], low[2];
    float slope2[2];
#pragma unroll
    for (int row = 0; row < 2; ++row) {
        mr[row] = warp * 16 + (lane >> 2) + 8 * row;
        const int tok = mr[row] / hg;
        pp[row] = tok < n ? pos0 + tok : -1;                      // -1: an idle row sees nothing
        low[row] = tok < n ? attn_low(p, pos0 + tok) : 0;
        slope2[row] = p.slope ? p.slope[g * hg + mr[row] % hg] * kLog2e : 0.f;
    }
    // positions this warp's rows span: tiles outside their windows are skipped
    const int wfirst = pos0 + min((warp * 16) / hg, n - 1), wlast = pos0 + min((warp * 16 + 15) / hg, n - 1);
    const int wlow = attn_low(p, wfirst);
    const bool wlive = (warp * 16) / hg < n;
    issue(0);
    for (int tile = 0; tile < ntile; ++tile) {
        issue(tile + 1);
        cp_wait<1>();
        __syncthreads();
        const int k0 = lo + tile * kPreKeys;
        if (wlive && k0 <= wlast && k0 + kPreKeys - 1 >= wlow) {
            const bf16* dk_ = skv + (size_t)(tile & 1) * kPreKeys * (ldk + ldv);
            const float* tab[2] = {nullptr, nullptr};
            if constexpr (BIAS) {
                const int ldb = attn_bias_ld(tq), d0 = pos0 - k0 - (kPreKeys - 1);
#pragma unroll
                for (int row = 0; row < 2; ++row) tab[row] = sbias + ((tile & 1) * hg + mr[row] % hg) * ldb - d0;      // read at seen distances only
            }
            attn_tiles<NV, kPreKeys / 16, BIAS>(sq + warp * 16 * ldk, ldk, dk_, ldk, dk_ + kPreKeys * ldk, ldv, p.dkp, k0, pos_last + 1, pp, low,
                                                p.scale * kLog2e, slope2, tab, 0, m, l, o);
        }
        __syncthreads();                                          // the buffer is refilled next
    }
    cp_wait<0>();
#pragma unroll
    for (int row = 0; row < 2; ++row) {
        l[row] += __shfl_xor_sync(0xffffffffu, l[row], 1);
        l[row] += __shfl_xor_sync(0xffffffffu, l[row], 2);
        const int tok = mr[row] / hg, h = g * hg + mr[row] % hg;
        if (tok >= n) continue;
        const size_t rr = (size_t)(r0 + tok);
        const float norm = attn_inv_sum(p, h, m[row], l[row]);
        if (p.out32) {
            float* d = p.out32 + (rr * p.H + h) * p.dvp + (lane & 3) * 2;
#pragma unroll
            for (int i = 0; i < NV; ++i) *reinterpret_cast<float2*>(d + i * 8) = make_float2(o[i][2 * row] * norm, o[i][2 * row + 1] * norm);
            continue;
        }
        const float inv = (p.off_gate >= 0 && p.head_gate ? gate_sigmoid(p.proj[rr * p.ldp + p.off_gate + h]) : 1.f) * p.out_scale * norm;
        bf16* d = reinterpret_cast<bf16*>(p.out) + rr * p.ldo + (size_t)h * p.dv;
        const float* gt = p.proj + rr * p.ldp + p.off_gate + (size_t)h * p.dv;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int c = i * 8 + (lane & 3) * 2 + u;
                if (c < p.dv) {
                    float v = o[i][2 * row + u] * inv;
                    if (p.off_gate >= 0 && !p.head_gate) v *= gate_sigmoid(gt[c]);
                    d[c] = __float2bfloat16(v);
                }
            }
    }
}

// the few-row form takes both maps of a differential head at once when its stages with both maps' keys fit an SM
static bool two_map_form(int maps, int dkp, int dvp) { return maps == 2 && (16 * (dkp + 8) + 4 * kDecStages * 16 * (2 * (dkp + 8) + dvp + 8)) * 2 <= 224 * 1024; }
template <int DVP>
static int launch_decode(const AttnParams& p, cudaStream_t st) {
    const int ldk = p.dkp + 8, ldv = DVP + 8;
    const bool both = two_map_form(p.maps, p.dkp, DVP) && !p.bias;
    size_t smem = (size_t)(16 * ldk + 4 * kDecStages * 16 * ((both ? 2 : 1) * ldk + ldv)) * 2;
    const size_t merge = (size_t)4 * 16 * (DVP + 2) * 4;
    if (merge > smem) smem = merge;
    static bool attr = false;
    if (!attr) {
        cudaFuncSetAttribute(attn_decode_kernel<DVP, 0, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        cudaFuncSetAttribute(attn_decode_kernel<DVP, 1, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        cudaFuncSetAttribute(attn_decode_kernel<DVP, 0, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        attr = true;
    }
    const dim3 grid(p.rows * p.G, p.NS, (p.H / p.G + 15) / 16);
    if (both) launch_pdl((attn_decode_kernel<DVP, 0, 2>), dim3(p.rows * (p.G / 2), p.NS, (p.H / p.G + 7) / 8), 128, smem, st, p);
    else if (p.bias) launch_pdl((attn_decode_kernel<DVP, 1, 1>), grid, 128, smem, st, p);
    else launch_pdl((attn_decode_kernel<DVP, 0, 1>), grid, 128, smem, st, p);
    if (p.NS > 1 && p.maps == 1) launch_pdl((attn_combine_kernel), dim3(p.rows, p.H), 128, 0, st, p);
    return (int)cudaGetLastError();
}
template <int DVP>
static int launch_prefill(const AttnParams& p, const int* row0, const int* nrows, int nseq, cudaStream_t st) {
    const int ldk = p.dkp + 8, ldv = DVP + 8, tq = 128 / (p.H / p.G);
    const size_t smem = (size_t)(128 * ldk + 2 * kPreKeys * (ldk + ldv)) * 2, sb = (size_t)2 * (p.H / p.G) * attn_bias_ld(tq) * 4;
    static bool attr = false;
    if (!attr) {
        cudaFuncSetAttribute(attn_prefill_kernel<DVP, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        cudaFuncSetAttribute(attn_prefill_kernel<DVP, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        attr = true;
    }
    const dim3 grid(p.rows / tq + nseq, p.G);
    if (p.bias) launch_pdl((attn_prefill_kernel<DVP, 1>), grid, 256, smem + sb, st, p, row0, nrows, nseq, tq);
    else launch_pdl((attn_prefill_kernel<DVP, 0>), grid, 256, smem, st, p, row0, nrows, nseq, tq);
    return (int)cudaGetLastError();
}

static bool tensor_form(int dkp, int dvp, int f32) { return !f32 && dkp <= 256 && dvp <= 256; }
static bool few_row_form(int run_rows, int H, int G, int dkp, int dvp, int f32) { return tensor_form(dkp, dvp, f32) && (run_rows < 8 || H / G > 128); }

}  // namespace lsb
using namespace lsb;

// Split sums per (row, head) that lsb_attn leaves to lsb_attn_diff in a step with runs of up to run_rows rows (1: normalised results).
LSB_API int lsb_attn_partials(int run_rows, int H, int G, int dkp, int dvp, int NS, int f32) { return few_row_form(run_rows, H, G, dkp, dvp, f32) ? NS : 1; }
// Blocks of the few-row form per row and key split
LSB_API int lsb_attn_blocks(int H, int G, int maps, int dkp, int dvp) {
    return two_map_form(maps, dkp, dvp) ? G / 2 * ((H / G + 7) / 8) : G * ((H / G + 15) / 16);
}
// padded head width of the cache and of the query buffer
LSB_API int lsb_attn_head_pad(int d) { return d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : (d + 127) / 128 * 128)); }

// Query / key norms (wq / wk null: none), value mixing (mix 0 none, 1 store v_first, 2 mix with lambda) and the cache append of every row.
LSB_API int lsb_attn_prep(const void* proj, int ldp, int off_q, int off_k, int off_v, const void* wq, const void* wk, float eps, void* vfirst, int mix,
                          const void* lambda, void* q_out, void* cache, const void* block_table, int max_pages, const void* row_seq, const void* row_pos,
                          int rows, int H, int G, int dk, int dv, int dkp, int dvp, int page, int f32, void* stream) {
    if (H % G || dkp < dk || dvp < dv || dkp % 16 || dvp % 16 || (mix && !vfirst) || (mix == 2 && !lambda)) return -1;
    cudaStream_t st = (cudaStream_t)stream;
    const bool wide = rows <= 64 && (H + 2 * G) * dk >= 2048;                   // few rows: a row's latency counts, not the blocks per SM
#define LSB_PREP(T, N) launch_pdl((attn_prep_kernel<T, N>), rows, N, 0, st, (const float*)proj, ldp, off_q, off_k, off_v, (const float*)wq, (const float*)wk, eps, \
                               (float*)vfirst, mix, (const float*)lambda, (T*)q_out, (T*)cache, (const int*)block_table, max_pages, (const int*)row_seq, \
                               (const int*)row_pos, H, G, dk, dv, dkp, dvp, page)
    if (f32) LSB_PREP(float, 256); else if (wide) LSB_PREP(bf16, 1024); else LSB_PREP(bf16, 256);
#undef LSB_PREP
    LSB_CHECK_LAUNCH();
}

// Biases (null: none), per-head norms (norm 0 none, 1 plain, 2 with wq / wk [dk]), rotation of the leading `rot` channels (inv_freq: fp64 [rot / 2]; pairs:
// adjacent channels, else halves), a factor per query head (temp, null: none) and the cache append of every row.  maps: see attn_head_prep_kernel.
LSB_API int lsb_attn_head_prep(const void* proj, int ldp, int off_q, int off_k, int off_v, const void* bias_q, const void* bias_k, const void* bias_v, int norm,
                               const void* wq, const void* wk, float eps, int rot, int pairs, const void* inv_freq, const void* temp, int maps, void* q_out, void* cache, const void* block_table,
                               int max_pages, const void* row_seq, const void* row_pos, int rows, int H, int G, int dk, int dv, int dkp, int dvp, int page,
                               int f32, void* stream) {
    if (rows < 1 || H % G || dkp < dk || dvp < dv || dkp % 16 || dvp % 16 || rot < 0 || rot % 2 || rot > dk || (rot && !inv_freq) || norm < 0 || norm > 2 ||
        (norm == 2 && (!wq || !wk)) || rot > 8192 || maps < 1 || G % maps)
        return -1;
    cudaStream_t st = (cudaStream_t)stream;
    const bool wide = rows <= 64 && H + 2 * G >= 12;
#define LSB_PREP(T, N) launch_pdl((attn_head_prep_kernel<T, N>), rows, N, (size_t)rot * 4, st, (const float*)proj, ldp, off_q, off_k, off_v, (const float*)bias_q, \
                               (const float*)bias_k, (const float*)bias_v, norm, (const float*)wq, (const float*)wk, eps, rot, pairs, (const double*)inv_freq, (const float*)temp, maps, (T*)q_out, \
                               (T*)cache, (const int*)block_table, max_pages, (const int*)row_seq, (const int*)row_pos, H, G, dk, dv, dkp, dvp, page)
    if (f32) LSB_PREP(float, 256); else if (wide) LSB_PREP(bf16, 1024); else LSB_PREP(bf16, 256);
#undef LSB_PREP
    LSB_CHECK_LAUNCH();
}

// Attention of the step's rows.  run_rows: the largest number of rows a sequence has in this step (host knowledge; it selects the kernel form).
// NS: key splits of the few-row form (o_part / ml_part sized for it).  off_gate < 0: no output gate; head_gate: one gate per head.  slope null: no linear
// distance bias; bias [H, bias_len] (null: none): learned distance bias, not together with slopes.  chunk: size of the mask's chunks (0: none).
// sink [H] (null: none).  maps > 1 (H and G count maps): the results stay in o_part for lsb_attn_diff, as split sums (NS > 1 and the few-row form) or
// normalised ([rows, H, dvp]).
LSB_API int lsb_attn(const void* q, const void* cache, const void* block_table, int max_pages, int page, const void* row_seq, const void* row_pos,
                     const void* seq_row0, const void* seq_nrows, int nseq, int run_rows, const void* proj, int ldp, int off_gate, void* out, int ldo,
                     void* o_part, void* ml_part, int NS, int rows, int H, int G, int dk, int dv, int dkp, int dvp, int window, float scale,
                     const void* slope, int head_gate, int chunk, const void* bias, int bias_len, float out_scale, const void* sink, int maps, int f32,
                     void* stream) {
    if (rows < 1 || H % G || dkp % 16 || dvp % 16 || NS < 1 || (NS > 1 && (!o_part || !ml_part)) || chunk < 0 || (bias && (slope || bias_len < 1)) ||
        maps < 1 || G % maps || (maps > 1 && (!o_part || sink)))
        return -1;
    AttnParams p;
    p.chunk = chunk; p.bias = (const float*)bias; p.bias_len = bias_len; p.out_scale = out_scale;
    p.q = q; p.cache = cache; p.block_table = (const int*)block_table; p.max_pages = max_pages; p.page = page; p.row_seq = (const int*)row_seq;
    p.row_pos = (const int*)row_pos; p.proj = (const float*)proj; p.ldp = ldp; p.off_gate = off_gate; p.head_gate = head_gate; p.out = out; p.ldo = ldo;
    p.o_part = (float*)o_part; p.ml_part = (float*)ml_part; p.rows = rows; p.H = H; p.G = G; p.dk = dk; p.dv = dv; p.dkp = dkp; p.dvp = dvp;
    p.maps = maps; p.sink = (const float*)sink; p.out32 = maps > 1 ? (float*)o_part : nullptr;
    p.ldc = G * dkp + G / maps * dvp; p.off_v = G * dkp; p.dkh = dkp; p.off_ks = 0; p.NS = NS; p.window = window; p.scale = scale; p.slope = (const float*)slope;
    cudaStream_t st = (cudaStream_t)stream;
    const bool tc = tensor_form(dkp, dvp, f32);
    const bool prefill = tc && !few_row_form(run_rows, H, G, dkp, dvp, f32);
    if (!tc) {
        const size_t smem = (size_t)(dkp + 256 + dv) * 4;
        if (smem > 48 * 1024) return -1;
        if (f32) launch_pdl((attn_exact_kernel<float>), dim3(rows, H), 128, smem, st, p);
        else launch_pdl((attn_exact_kernel<bf16>), dim3(rows, H), 128, smem, st, p);
        LSB_CHECK_LAUNCH();
    }
    switch (dvp) {
        case 32: return prefill ? launch_prefill<32>(p, (const int*)seq_row0, (const int*)seq_nrows, nseq, st) : launch_decode<32>(p, st);
        case 64: return prefill ? launch_prefill<64>(p, (const int*)seq_row0, (const int*)seq_nrows, nseq, st) : launch_decode<64>(p, st);
        case 128: return prefill ? launch_prefill<128>(p, (const int*)seq_row0, (const int*)seq_nrows, nseq, st) : launch_decode<128>(p, st);
        case 256: return prefill ? launch_prefill<256>(p, (const int*)seq_row0, (const int*)seq_nrows, nseq, st) : launch_decode<256>(p, st);
    }
    return -1;
}

// Differential heads from what lsb_attn (maps = 2) left in parts: H query heads in groups of hg, out [rows, ldo] heads side by side.  NS: split sums per map
// (with ml) or 1 (ml null: normalised results).
LSB_API int lsb_attn_diff(void* out, int ldo, const void* parts, const void* ml, int NS, int rows, int H, int hg, int dv, int dvp, float lambda, float eps, float factor,
                          const void* row_seq, int f32, void* stream) {
    if (rows < 1 || H < 1 || hg < 1 || H % hg || NS < 1 || NS > 32 || (NS > 1 && !ml) || dv < 1 || dv > dvp || dv > 3000) return -1;
    cudaStream_t st = (cudaStream_t)stream;
    const int nq = (dv + 3) / 4;
    int ng = 256 / nq;
    ng = ng < 1 ? 1 : (ng < NS ? ng : NS);
#define LSB_AD(T)                                                                                                                                                    \
    if (NS > 1) launch_pdl((attn_diff_merge_kernel<T>), dim3(rows, H), 256, (size_t)ng * nq * 16, st, (T*)out, ldo, (const float*)parts, (const float*)ml, NS, ng, H, hg,  \
                           dv, dvp, lambda, eps, factor, (const int*)row_seq);                                                                                       \
    else launch_pdl((attn_diff_kernel<T>), dim3(rows, (H + 3) / 4), 128, (size_t)16 * dv, st, (T*)out, ldo, (const float*)parts, H, hg, dv, dvp, lambda, eps, factor,      \
                    (const int*)row_seq)
    if (f32) { LSB_AD(float); } else { LSB_AD(bf16); }
#undef LSB_AD
    LSB_CHECK_LAUNCH();
}

// Attention of one run of rows (positions row_pos, causal, sliding window or 0) over keys and values written out per head and position: kv [positions, H dkh keys | H dvp values |
// dks key channels shared by all heads].  q: [rows, H, dkh + dks].  seq_row0 / seq_nrows: the run, as the other kernels take it; page0: a zero (the rows
// are one page; the first is position key_base); off_gate: one gate per head (head_gate) or value channel (-1: none).
LSB_API int lsb_attn_run(const void* q, const void* kv, int positions, const void* page0, const void* row_seq, const void* row_pos, const void* seq_row0,
                         const void* seq_nrows, const void* proj, int ldp, int off_gate, int head_gate, void* out, int ldo, int rows, int H, int dkh, int dks, int dv,
                         int dvp, int window, int key_base, float scale, void* stream) {
    if (key_base < 0 || rows < 1 || dkh % 16 || dks % 16 || dkh + dks > 256 || dv > dvp) return -1;
    AttnParams p;
    p.q = q; p.cache = kv; p.block_table = (const int*)page0; p.max_pages = 0; p.page = positions; p.row_seq = (const int*)row_seq; p.row_pos = (const int*)row_pos;
    p.proj = (const float*)proj; p.ldp = ldp; p.off_gate = off_gate; p.head_gate = head_gate; p.out = out; p.ldo = ldo; p.o_part = p.ml_part = nullptr; p.rows = rows;
    p.key_base = key_base; p.H = p.G = H; p.dk = p.dkp = dkh + dks; p.dv = dv; p.dvp = dvp; p.dkh = dkh; p.off_ks = H * (dkh + dvp); p.ldc = H * (dkh + dvp) + dks; p.off_v = H * dkh;
    p.NS = 1; p.window = window; p.scale = scale; p.slope = nullptr;
    switch (dvp) {
        case 32: return launch_prefill<32>(p, (const int*)seq_row0, (const int*)seq_nrows, 1, (cudaStream_t)stream);
        case 64: return launch_prefill<64>(p, (const int*)seq_row0, (const int*)seq_nrows, 1, (cudaStream_t)stream);
        case 128: return launch_prefill<128>(p, (const int*)seq_row0, (const int*)seq_nrows, 1, (cudaStream_t)stream);
        case 256: return launch_prefill<256>(p, (const int*)seq_row0, (const int*)seq_nrows, 1, (cudaStream_t)stream);
    }
    return -1;
}

LSB_API int lsb_trace_set_attn(void* buf) { return lsb_trace_install(buf); }
