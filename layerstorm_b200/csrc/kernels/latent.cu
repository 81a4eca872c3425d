// Latent attention over the paged cache, absorbed form, for models described layer by layer: one cached row [latent | rotated key part] per
// token serves every head, whole causal prefix or a sliding window, fp32 scores and weights, an output gate per head or per value channel.  All sizes
// are run-time parameters; the rotated part may be missing.
//
//   c = RMSNorm(y[:dl]),  k_r = rot(y[dl:])                     y: the layer's latent projection (none: another layer's rows are read)
//   q'_h = [ W_uk,h^T q_h | rot(q_r,h) ]                        the unrotated query moved into the latent space
//   s_ij = scale q'_i . [c_j | k_r,j],  o_i = sum_j softmax_j(s_ij) c_j
//   out_h = W_uv,h (sigmoid(g_h) o_h), or sigmoid(g_h) * (W_uv,h o_h) with a gate per value channel
//
// Rotary pairs are adjacent channels.  Cache row of a token: [dlp latent | drp rotated], widths padded with zeros to multiples of 16.
//   latent_query    few rows (and fp32): rotation, absorption and the cache append in one launch
//   latent_prep     many rows: rotation, append and the bf16 operand of the absorbing product, which then runs on the tcgen05 GEMM
//   latent_attn     (token, head) rows of a sequence in tiles of 16 MG against key tiles shared by all of them; any mixture of prompt runs and
//                   single tokens; key splits for small batches: up to eight splits are a thread-block cluster that merges its sums through
//                   distributed shared memory, what is left (one partial sum per cluster) goes through global memory
//   latent_rows / latent_gather   long runs of one sequence: keys and values are written out per head for all its positions (one tcgen05
//                   product over the gathered latents; the rotated part stays shared), and the run goes through the grouped-query prefill kernel (attn.cu) - a third of the
//                   arithmetic per (query, key) of the absorbed form, for products that do not depend on the number of queries
//   latent_combine  merge of those partial sums;  latent_out: the same together with the value up-projection (few rows)
// The value of a key is the head of its cache row, so a key tile is loaded once for both products.
#include "attn_core.cuh"
#include <cooperative_groups.h>

extern "C" int lsb_gemm_bf16_tc_batched(void* out, const void* x, const void* w, int M, int N, int K, int B, int ldx, long long xs_b, int ldw,
                                        long long ws_b, int ldo, long long os_b, int out_bf16, void* err, void* stream);
extern "C" int lsb_gemm_bf16_tc(void* out, const void* x, const void* w, const void* bias, int M, int N, int K, int ldx, int ldw, int ldo, int out_bf16,
                                void* partial, long long partial_cap, void* err, const void* comm, void* stream);

namespace lsb {
namespace cg = cooperative_groups;

struct LatentPrep {
    const float* qsrc; int ldq;                       // queries, from their first column on
    const float* proj; int ldp, off_kv;               // off_kv < 0: the layer has no latent projection of its own
    const float* kv_norm; float eps;
    const double* inv_freq;                           // [dr / 2]
    const void* w_uk;                                 // [H, dlp, dnp]
    void* q;                                          // [rows, H, dlp + drp]
    bf16* q_nope;                                     // [rows, H, dnp] (many-row form)
    void* cache; const int* block_table; int max_pages, page;
    const int* row_seq; const int* row_pos;
    int rows, H, dn, dnp, dr, drp, dl, dlp;
};

// (a, b) turned by pos * freq
__device__ __forceinline__ void rotate_pair(float& a, float& b, int pos, double freq) {
    float s, c;
    rotary_angle(pos, freq, s, c);
    const float u = a * c - b * s, v = b * c + a * s;
    a = u; b = v;
}

template <typename T>
__device__ __forceinline__ void rotated_tail(T* dst, const float* src, int dr, int drp, int pos, const double* inv_freq, int t, int nt) {
    for (int i = t; i < drp / 2; i += nt) {
        float a = 0.f, b = 0.f;
        if (2 * i < dr) { a = src[2 * i]; b = src[2 * i + 1]; rotate_pair(a, b, pos, inv_freq[i]); }
        dst[2 * i] = to_act<T>(a); dst[2 * i + 1] = to_act<T>(b);
    }
}

// Whole block: latent norm, rotation, append of row r.
template <typename T>
__device__ __forceinline__ void append_row(const LatentPrep& p, int r, float* red) {
    const int t = threadIdx.x, nt = blockDim.x, seq = p.row_seq[r], pos = p.row_pos[r];
    const float* y = p.proj + (size_t)r * p.ldp + p.off_kv;
    float ss = 0.f;
    for (int i = t; i < p.dl; i += nt) { const float v = y[i]; ss = fmaf(v, v, ss); }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.dl + p.eps);
    if (seq < 0) return;
    T* row = reinterpret_cast<T*>(p.cache) + ((size_t)p.block_table[(size_t)seq * p.max_pages + pos / p.page] * p.page + pos % p.page) * (p.dlp + p.drp);
    for (int i = t; i < p.dlp; i += nt) row[i] = to_act<T>(i < p.dl ? y[i] * inv * p.kv_norm[i] : 0.f);
    rotated_tail(row + p.dlp, y + p.dl, p.dr, p.drp, pos, p.inv_freq, t, nt);
}

template <typename T> struct Vec16 { static constexpr int N = 16 / (int)sizeof(T); };
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[8]) { unpack_bf16x8(v, f); }
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[4]) {
    f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
}

// Rows n0 .. n1 of a [.., K] matrix against MT fp32 vectors in shared memory (K a multiple of 8): a group of lanes per matrix row, 16 bytes per
// lane; emit(n, sums) runs on one lane of the group.  Whole block of 256 threads.
template <typename T, int MT, typename Emit>
__device__ __forceinline__ void small_products(const T* w, int K, int n0, int n1, const float* xs, int ldx, Emit emit) {
    constexpr int V = Vec16<T>::N;
    int lg = 1;
    while (lg < 32 && lg * V < K) lg <<= 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = 32 / lg, sub = lane / lg, l0 = lane & (lg - 1);
#pragma unroll 4
    for (int nb = n0 + warp * per; nb < n1; nb += 8 * per) {
        const int n = min(nb + sub, n1 - 1);
        float acc[MT];
#pragma unroll
        for (int m = 0; m < MT; ++m) acc[m] = 0.f;
        for (int k = l0 * V; k < K; k += lg * V) {
            float f[V];
            unpack16(ldg_stream(w + (size_t)n * K + k), f);
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int e = 0; e < V; ++e) acc[m] = fmaf(f[e], xs[m * ldx + k + e], acc[m]);
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
            for (int o = lg >> 1; o > 0; o >>= 1) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
        if (l0 == 0 && nb + sub < n1) emit(n, acc);
    }
}

// Weights do not depend on the previous kernel: on their way to L2 before the dependency wait (first block of a column range only).
template <typename T>
__device__ __forceinline__ void prefetch_rows(const T* w, size_t n) {
    if (blockIdx.z) return;
    const char* b = reinterpret_cast<const char*>(w);
    for (size_t i = (size_t)threadIdx.x * 128; i < n * sizeof(T); i += 256 * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(b + i));
}

constexpr int kQueryCols = 128;       // latent columns per block of latent_query
template <typename T, int MT>
__global__ void __launch_bounds__(256) latent_query_kernel(LatentPrep p) {
    extern __shared__ __align__(16) float lsm[];              // [MT][dnp]
    __shared__ float red[33];
    const int h = blockIdx.y, r0 = blockIdx.z * MT, nr = min(MT, p.rows - r0), t = threadIdx.x, D = p.dlp + p.drp;
    const int n0 = blockIdx.x * kQueryCols, n1 = min(p.dlp, n0 + kQueryCols);
    if (n0 < n1) prefetch_rows(reinterpret_cast<const T*>(p.w_uk) + ((size_t)h * p.dlp + n0) * p.dnp, (size_t)(n1 - n0) * p.dnp);
    pdl_wait();
    pdl_launch_dependents();
    T* q = reinterpret_cast<T*>(p.q) + ((size_t)r0 * p.H + h) * D;
    const float* src = p.qsrc + (size_t)r0 * p.ldq + (size_t)h * (p.dn + p.dr);
    if (blockIdx.x == gridDim.x - 1) {                        // rotations of this head; row m's append falls to head m
        for (int m = 0; m < nr; ++m)
            rotated_tail(q + (size_t)m * p.H * D + p.dlp, src + (size_t)m * p.ldq + p.dn, p.dr, p.drp, p.row_pos[r0 + m], p.inv_freq, t, 256);
        if (p.off_kv >= 0)
            for (int m = h; m < nr; m += p.H) append_row<T>(p, r0 + m, red);
        return;
    }
    for (int i = t; i < MT * p.dnp; i += 256) {
        const int m = i / p.dnp, c = i - m * p.dnp;
        lsm[i] = m < nr && c < p.dn ? src[(size_t)m * p.ldq + c] : 0.f;
    }
    __syncthreads();
    small_products<T, MT>(reinterpret_cast<const T*>(p.w_uk) + (size_t)h * p.dlp * p.dnp, p.dnp, n0, n1, lsm, p.dnp, [&](int n, const float (&a)[MT]) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
            if (m < nr) q[(size_t)m * p.H * D + n] = to_act<T>(a[m]);
    });
}

// Rotated parts of all heads of a row (dst: rows of ld, src: rows of dn + dr); a thread keeps its rotary pair over the heads: one angle per pair.
__device__ __forceinline__ void rotated_heads(bf16* dst, int ld, const float* src, const LatentPrep& p, int pos, int hp) {
    if (hp == 0) return;
    const int t = threadIdx.x, w = min(hp, 256), step = 256 / w, h0 = t / w;
    for (int i = h0 < step ? t % w : hp; i < hp; i += w) {
        float cs = 1.f, sn = 0.f;
        if (2 * i < p.dr) rotate_pair(cs, sn, pos, p.inv_freq[i]);
        for (int h = h0; h < p.H; h += step) {
            float a = 0.f, b = 0.f;
            if (2 * i < p.dr) { const float* s = src + (size_t)h * (p.dn + p.dr) + 2 * i; a = s[0]; b = s[1]; }
            *reinterpret_cast<bf162*>(dst + (size_t)h * ld + 2 * i) = __floats2bfloat162_rn(a * cs - b * sn, b * cs + a * sn);
        }
    }
}

__global__ void __launch_bounds__(256) latent_prep_kernel(LatentPrep p) {
    __shared__ float red[33];
    const int r = blockIdx.x, t = threadIdx.x, D = p.dlp + p.drp, hp = p.drp / 2;
    pdl_wait();
    pdl_launch_dependents();
    const int pos = p.row_pos[r];
    const float* src = p.qsrc + (size_t)r * p.ldq;
    bf16* qn = p.q_nope + (size_t)r * p.H * p.dnp;
    if (p.dn == p.dnp && ((p.dn + p.dr) | p.ldq) % 4 == 0 && (reinterpret_cast<uintptr_t>(p.qsrc) & 15) == 0) {
        const int n4 = p.dn / 4;
        for (int i = t; i < p.H * n4; i += 256) {
            const int h = i / n4, c = (i - h * n4) * 4;
            const float4 v = *reinterpret_cast<const float4*>(src + (size_t)h * (p.dn + p.dr) + c);
            bf162* d = reinterpret_cast<bf162*>(qn + (size_t)h * p.dnp + c);
            d[0] = __floats2bfloat162_rn(v.x, v.y); d[1] = __floats2bfloat162_rn(v.z, v.w);
        }
    } else {
        for (int i = t; i < p.H * p.dnp; i += 256) {
            const int h = i / p.dnp, c = i - h * p.dnp;
            qn[i] = __float2bfloat16(c < p.dn ? src[(size_t)h * (p.dn + p.dr) + c] : 0.f);
        }
    }
    rotated_heads(reinterpret_cast<bf16*>(p.q) + (size_t)r * p.H * D + p.dlp, D, src + p.dn, p, pos, hp);
    if (p.off_kv >= 0) append_row<bf16>(p, r, red);
}

// ------------------------------------------------------------------------------------------------ keys and values written out per head
// Row r: q [H, dnw + drp] (unrotated part padded to dnw, rotated part behind it), cache append.
__global__ void __launch_bounds__(256) latent_rows_kernel(LatentPrep p, int dnw) {
    __shared__ float red[33];
    const int r = blockIdx.x, t = threadIdx.x, K = dnw + p.drp, hp = p.drp / 2;
    pdl_wait();
    pdl_launch_dependents();
    const int pos = p.row_pos[r];
    const float* src = p.qsrc + (size_t)r * p.ldq;
    bf16* q = reinterpret_cast<bf16*>(p.q) + (size_t)r * p.H * K;
    for (int i = t; i < p.H * (dnw / 2); i += 256) {
        const int h = i / (dnw / 2), c = (i - h * (dnw / 2)) * 2;
        const float* s = src + (size_t)h * (p.dn + p.dr) + c;
        *reinterpret_cast<bf162*>(q + (size_t)h * K + c) = __floats2bfloat162_rn(c < p.dn ? s[0] : 0.f, c + 1 < p.dn ? s[1] : 0.f);
    }
    rotated_heads(q + dnw, K, src + p.dn, p, pos, hp);
    if (p.off_kv >= 0) append_row<bf16>(p, r, red);
}

// Cached rows of positions [base, T) of one sequence: the latents to lat [T - base, dlp], the rotated part to column off_rot of kv's rows.  One warp per position.
__global__ void __launch_bounds__(128) latent_gather_kernel(const bf16* __restrict__ cache, const int* __restrict__ block_table, int max_pages, int page,
                                                            const int* __restrict__ row_seq, int base, int T, int dlp, int drp, bf16* __restrict__ lat,
                                                            bf16* __restrict__ kv, int ldkv, int off_rot) {
    const int j = base + blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    pdl_wait();
    pdl_launch_dependents();
    const int seq = row_seq[0];
    if (seq < 0 || j >= T) return;
    const uint4* src = reinterpret_cast<const uint4*>(cache + ((size_t)block_table[(size_t)seq * max_pages + j / page] * page + j % page) * (dlp + drp));
    for (int i = lane; i < (dlp + drp) / 8; i += 32) {
        if (i < dlp / 8) reinterpret_cast<uint4*>(lat + (size_t)(j - base) * dlp)[i] = src[i];
        else reinterpret_cast<uint4*>(kv + (size_t)(j - base) * ldkv + off_rot)[i - dlp / 8] = src[i];
    }
}

// ------------------------------------------------------------------------------------------------ attention (mma.sync m16n8k16)
struct LatentAttn {
    const bf16* q;                    // [rows, H, D]
    const bf16* cache; const int* block_table; int max_pages, page;
    const int* row_seq; const int* row_pos; const int* seq_row0; const int* seq_nrows; int nseq, run_rows;
    const float* proj; int ldp, off_gate;
    bf16* out;                        // [rows, H, dlp]
    float* o_part; float* ml_part;    // [rows, H, NS / C, dlp], [rows, H, NS / C, 2]
    int H, dlp, drp, window, NS, C;   // sliding window (0: none), key splits, and how many of them form a cluster
    float scale2;                     // log2 units
};

// NV: 8-column value tiles per warp (latent width up to 64 NV); MG: 16-row tiles of (token, head) rows per block
template <int NV, int MG> struct LatentCfg {
    static constexpr int BM = MG * 16, KT = MG == 4 ? 32 : 64, STAGES = MG == 4 ? 3 : 2;
    static constexpr int RANGES = 8 / MG, KW = KT / RANGES, NT = KW / 8, LDP = KT + 8;      // score phase: a warp owns 16 rows x KW keys
    static __host__ __device__ int ld(int D) { return (D > NV * 64 ? D : NV * 64) + 8; }     // an odd multiple of 16 bytes
    static size_t smem(int D) { return (size_t)(BM + STAGES * KT) * ld(D) * 2 + (size_t)2 * BM * LDP * 2 + (size_t)(RANGES + 1) * BM * 4; }
    // the cluster merge reuses the query and key tiles
    static_assert((size_t)BM * (NV * 64 + 4) * 4 + 8 * BM * 4 <= (size_t)(BM + STAGES * KT) * (NV * 64 + 8) * 2, "merge scratch");
};
__device__ __forceinline__ void ldsm2(uint32_t (&r)[2], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(sm_addr(p)));
}
__device__ __forceinline__ void ldsm2_t(uint32_t (&r)[2], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(sm_addr(p)));
}

template <int NV, int MG>
__global__ void __launch_bounds__(256, 1) latent_attn_kernel(LatentAttn p) {
    using C = LatentCfg<NV, MG>;
    constexpr int BM = C::BM, KT = C::KT, NT = C::NT, LDP = C::LDP;
    extern __shared__ __align__(16) bf16 asm_[];
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, D = p.dlp + p.drp, ld = C::ld(D);
    bf16* sq = asm_;                                              // [BM][ld]
    bf16* sk = sq + BM * ld;                                      // [STAGES][KT][ld]
    bf16* sph = sk + C::STAGES * KT * ld;                         // [BM][LDP] weights, high parts
    bf16* spl = sph + BM * LDP;                                   // ... and remainders
    float* s_max = reinterpret_cast<float*>(spl + BM * LDP);      // [RANGES][BM]
    float* s_corr = s_max + C::RANGES * BM;                       // [BM]
    pdl_wait();
    pdl_launch_dependents();
    // block -> tokens [row0, row0 + n) of one sequence and the first (token, head) row f0 of its tile; late tiles (most keys) first
    int tile = (int)(gridDim.x - 1 - blockIdx.x), row0 = 0, n = 0, f0 = 0;
    if (p.run_rows == 1) {
        const int per = (p.H + BM - 1) / BM;
        row0 = tile / per; f0 = (tile - row0 * per) * BM; n = 1;
    } else {
        for (int s = 0; s < p.nseq; ++s) {
            const int ns = p.seq_nrows[s], nt = (ns * p.H + BM - 1) / BM;
            if (tile < nt) { row0 = p.seq_row0[s]; n = ns; f0 = tile * BM; break; }
            tile -= nt;
        }
        if (n == 0) return;
    }
    const int seq = p.row_seq[row0], pos0 = p.row_pos[row0];
    if (seq < 0) return;
    const int nf = min(BM, n * p.H - f0);                         // rows of the tile in use
    const int pos_first = pos0 + f0 / p.H, pos_last = pos0 + (f0 + nf - 1) / p.H;
    const int chunks = D / 8;
    for (int i = t; i < BM * chunks; i += 256) {
        const int m = i / chunks, c = i - m * chunks;
        if (m < nf) cp16(sq + m * ld + c * 8, p.q + ((size_t)row0 * p.H + f0 + m) * D + c * 8);
        else *reinterpret_cast<uint4*>(sq + m * ld + c * 8) = make_uint4(0, 0, 0, 0);
    }
    auto low = [&](int pos) { return p.window > 0 ? max(0, pos - p.window + 1) : 0; };          // first key that a position sees
    const int key0 = low(pos_first), ntile = (pos_last - key0) / KT + 1, per = (ntile + p.NS - 1) / p.NS, t0 = (int)blockIdx.y * per, t1 = min(ntile, t0 + per);
    constexpr int TPK = 256 / KT;                                 // threads per key of a tile copy
    const int kr = t / TPK;
    const int* bt = p.block_table + (size_t)seq * p.max_pages;
    auto locate = [&](int kt) {                                   // cache row of this thread's key in tile kt
        const int j = min(key0 + kt * KT + kr, pos_last);                // keys past the tile's last position are clamped (masked later)
        return kt < t1 ? (size_t)bt[j / p.page] * p.page + j % p.page : 0;
    };
    size_t ahead = locate(t0);                                    // looked up one tile early: the copies do not wait for the table
    auto issue = [&](int kt) {
        if (kt < t1) {
            const bf16* src = p.cache + ahead * D;
            bf16* dst = sk + ((size_t)((kt - t0) % C::STAGES) * KT + kr) * ld;
            for (int c = t % TPK; c < chunks; c += TPK) cp16(dst + c * 8, src + c * 8);
            ahead = locate(kt + 1);
        }
        cp_commit();
    };
    const int mi = warp % MG, ki = warp / MG;
    int pr[2], lo[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int m = mi * 16 + (lane >> 2) + 8 * u;
        pr[u] = m < nf ? pos0 + (f0 + m) / p.H : -1;              // -1: an idle row sees nothing
        lo[u] = low(pr[u]);
    }
    float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[MG][NV][4];
#pragma unroll
    for (int a = 0; a < MG; ++a)
#pragma unroll
        for (int b = 0; b < NV; ++b) { o[a][b][0] = o[a][b][1] = o[a][b][2] = o[a][b][3] = 0.f; }
#pragma unroll
    for (int s = 0; s < C::STAGES - 1; ++s) issue(t0 + s);
    const bf16* qp = sq + (mi * 16 + (lane & 15)) * ld + (lane >> 4) * 8;
    const int kofs = NT == 2 ? (ki * 16 + (lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8 : (ki * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
    const int vofs = ((lane & 7) + ((lane >> 3) & 1) * 8) * ld + warp * NV * 8 + (NV > 1 ? (lane >> 4) * 8 : 0);
    const int pofs = (lane & 15) * LDP + (lane >> 4) * 8;
    for (int kt = t0; kt < t1; ++kt) {
        cp_wait<C::STAGES - 2>();
        __syncthreads();                                          // the tile is in, the previous tile's buffer is free
        issue(kt + C::STAGES - 1);
        const bf16* kb = sk + (size_t)((kt - t0) % C::STAGES) * KT * ld;
        // ---- scores of 16 rows x KW keys; even and odd steps of the reduction in separate sums
        float s[2][NT][4];
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
            for (int b = 0; b < NT; ++b) s[a][b][0] = s[a][b][1] = s[a][b][2] = s[a][b][3] = 0.f;
        auto step = [&](int k, float (&acc)[NT][4]) {
            uint32_t a[4];
            ldsm4(a, qp + k);
            if constexpr (NT == 2) {
                uint32_t b[4];
                ldsm4(b, kb + kofs + k);
                mma_bf16(acc[0], a, b[0], b[1]);
                mma_bf16(acc[1], a, b[2], b[3]);
            } else {
                uint32_t b[2];
                ldsm2(b, kb + kofs + k);
                mma_bf16(acc[0], a, b[0], b[1]);
            }
        };
        int k = 0;
#pragma unroll(MG == 4 ? 2 : 4)
        for (; k + 32 <= D; k += 32) { step(k, s[0]); step(k + 16, s[1]); }
        if (k < D) step(k, s[0]);
        float mt[2] = {-INFINITY, -INFINITY};
        const bool full = key0 + kt * KT + KT - 1 <= pos_first && nf == BM && key0 + kt * KT >= low(pos_last);
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float v = (s[0][i][j] + s[1][i][j]) * p.scale2;
                const int key = key0 + kt * KT + ki * C::KW + i * 8 + (lane & 3) * 2 + (j & 1);
                s[0][i][j] = full || (key <= pr[j >> 1] && key >= lo[j >> 1]) ? v : -INFINITY;
                mt[j >> 1] = fmaxf(mt[j >> 1], s[0][i][j]);
            }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            mt[u] = fmaxf(mt[u], __shfl_xor_sync(0xffffffffu, mt[u], 1));
            mt[u] = fmaxf(mt[u], __shfl_xor_sync(0xffffffffu, mt[u], 2));
            if ((lane & 3) == 0) s_max[ki * BM + mi * 16 + (lane >> 2) + 8 * u] = mt[u];
        }
        __syncthreads();
        float base[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int row = mi * 16 + (lane >> 2) + 8 * u;
            float m = mx[u];
#pragma unroll
            for (int r = 0; r < C::RANGES; ++r) m = fmaxf(m, s_max[r * BM + row]);
            base[u] = m == -INFINITY ? 0.f : m;
            const float corr = ex2(mx[u] - base[u]);              // nothing seen yet: 0
            mx[u] = m;
            l[u] *= corr;
            if (ki == 0 && (lane & 3) == 0) s_corr[row] = corr;
        }
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float e0 = ex2(s[0][i][2 * u] - base[u]), e1 = ex2(s[0][i][2 * u + 1] - base[u]);
                l[u] += e0 + e1;
                uint32_t hi, lo;
                split2(e0, e1, hi, lo);
                const int at = (mi * 16 + (lane >> 2) + 8 * u) * LDP + ki * C::KW + i * 8 + (lane & 3) * 2;
                *reinterpret_cast<uint32_t*>(sph + at) = hi;
                *reinterpret_cast<uint32_t*>(spl + at) = lo;
            }
        __syncthreads();
        // ---- values: this warp's latent columns for all rows of the tile
        float c0[MG], c1[MG];
        bool keep = true;
#pragma unroll
        for (int a = 0; a < MG; ++a) {
            c0[a] = s_corr[a * 16 + (lane >> 2)]; c1[a] = s_corr[a * 16 + (lane >> 2) + 8];
            keep = keep && c0[a] == 1.f && c1[a] == 1.f;
        }
        if (!__all_sync(0xffffffffu, keep)) {
#pragma unroll
            for (int a = 0; a < MG; ++a)
#pragma unroll
                for (int b = 0; b < NV; ++b) { o[a][b][0] *= c0[a]; o[a][b][1] *= c0[a]; o[a][b][2] *= c1[a]; o[a][b][3] *= c1[a]; }
        }
#pragma unroll
        for (int ks = 0; ks < KT; ks += 16) {
            uint32_t v[NV][2];
            if constexpr (NV == 1) ldsm2_t(v[0], kb + vofs + ks * ld);
            else {
#pragma unroll
                for (int b = 0; b < NV; b += 2) {
                    uint32_t r[4];
                    ldsm4_t(r, kb + vofs + ks * ld + b * 8);
                    v[b][0] = r[0]; v[b][1] = r[1]; v[b + 1][0] = r[2]; v[b + 1][1] = r[3];
                }
            }
#pragma unroll
            for (int a = 0; a < MG; ++a) {
                uint32_t hi[4], lo[4];
                ldsm4(hi, sph + a * 16 * LDP + pofs + ks);
                ldsm4(lo, spl + a * 16 * LDP + pofs + ks);
#pragma unroll
                for (int b = 0; b < NV; ++b) { mma_bf16(o[a][b], hi, v[b][0], v[b][1]); mma_bf16(o[a][b], lo, v[b][0], v[b][1]); }
            }
        }
    }
    cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
        l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
        const int row = mi * 16 + (lane >> 2) + 8 * u;
        if ((lane & 3) == 0) {
            s_max[ki * BM + row] = l[u];
            if (ki == 0) s_corr[row] = mx[u];
        }
    }
    __syncthreads();
    float L = 0.f;
    if (t < BM) {
#pragma unroll
        for (int r = 0; r < C::RANGES; ++r) L += s_max[r * BM + t];
    }
    __syncthreads();
    if (t < BM) s_max[t] = L;                                     // sums and maxima of the tile's rows: s_max[m], s_corr[m]
    auto gate = [&](int m) {
        return p.off_gate >= 0 ? gate_sigmoid(p.proj[(size_t)(row0 + (f0 + m) / p.H) * p.ldp + p.off_gate + (f0 + m) % p.H]) : 1.f;
    };
    if (p.C == 1) {
        __syncthreads();
#pragma unroll
        for (int a = 0; a < MG; ++a)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int m = a * 16 + (lane >> 2) + 8 * u;
                if (m >= nf) continue;
                const size_t rh = (size_t)row0 * p.H + f0 + m;
                const float f = gate(m) / s_max[m];
#pragma unroll
                for (int b = 0; b < NV; ++b) {
                    const int c = (warp * NV + b) * 8 + (lane & 3) * 2;
                    if (c < p.dlp) *reinterpret_cast<bf162*>(p.out + rh * p.dlp + c) = __floats2bfloat162_rn(o[a][b][2 * u] * f, o[a][b][2 * u + 1] * f);
                }
            }
        return;
    }
    // merge inside the cluster: every CTA shows its sums, and takes an equal share of the columns of all of them
    constexpr int LDO = NV * 64 + 4;
    float* so = reinterpret_cast<float*>(asm_);                   // [BM][LDO], over the query and key tiles
    float* s_w = so + BM * LDO;                                   // [8][BM] weights of the CTAs, then the row's factor
#pragma unroll
    for (int a = 0; a < MG; ++a)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            float* d = so + (a * 16 + (lane >> 2) + 8 * u) * LDO + warp * NV * 8 + (lane & 3) * 2;
#pragma unroll
            for (int b = 0; b < NV; ++b) *reinterpret_cast<float2*>(d + b * 8) = make_float2(o[a][b][2 * u], o[a][b][2 * u + 1]);
        }
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    const int rank = (int)cluster.block_rank(), NSo = p.NS / p.C, so_i = (int)blockIdx.y / p.C;
    if (t < nf) {
        float mm[8], ll[8], M = -INFINITY;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            mm[j] = j < p.C ? cluster.map_shared_rank(s_corr, j)[t] : -INFINITY;
            ll[j] = j < p.C ? cluster.map_shared_rank(s_max, j)[t] : 0.f;
            M = fmaxf(M, mm[j]);
        }
        float S = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            mm[j] = mm[j] == -INFINITY ? 0.f : ex2(mm[j] - M);
            S = fmaf(mm[j], ll[j], S);
        }
        const float f = NSo == 1 ? gate(t) / S : 1.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) s_w[j * BM + t] = mm[j] * f;
        if (NSo > 1 && rank == 0) {
            const size_t k = ((size_t)row0 * p.H + f0 + t) * NSo + so_i;
            p.ml_part[2 * k] = M; p.ml_part[2 * k + 1] = S;
        }
    }
    __syncthreads();
    const int quads = NV * 16 / p.C;                              // groups of four columns per CTA
    for (int i = t; i < nf * quads; i += 256) {
        const int m = i / quads, c = (rank * quads + i - m * quads) * 4;
        float4 v[8], a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (j < p.C) v[j] = *reinterpret_cast<const float4*>(cluster.map_shared_rank(so, j) + m * LDO + c);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (j < p.C) { const float w = s_w[j * BM + m]; a.x = fmaf(w, v[j].x, a.x); a.y = fmaf(w, v[j].y, a.y); a.z = fmaf(w, v[j].z, a.z); a.w = fmaf(w, v[j].w, a.w); }
        if (c >= p.dlp) continue;
        const size_t rh = (size_t)row0 * p.H + f0 + m;
        if (NSo == 1) {
            bf162* d = reinterpret_cast<bf162*>(p.out + rh * p.dlp + c);
            d[0] = __floats2bfloat162_rn(a.x, a.y); d[1] = __floats2bfloat162_rn(a.z, a.w);
        } else {
            *reinterpret_cast<float4*>(p.o_part + (rh * NSo + so_i) * p.dlp + c) = a;
        }
    }
    cluster.sync();                                               // nobody leaves while its sums may still be read
}

// ------------------------------------------------------------------------------------------------ split merge, value up-projection
struct LatentOut {
    const void* o_lat;                // [rows, H, dlp], gated (NS == 1)
    const float* o_part; const float* ml_part; int NS;
    const float* proj; int ldp, off_gate, head_gate;      // gate per head (of the latent sums) or per value channel (of the result)
    const int* row_seq;
    int rows, H, dlp, dv;
};
// One warp: weights (with the gate and the softmax sum folded in) of the splits of row r, head h.
__device__ __forceinline__ void split_weights(const LatentOut& p, int r, int h, float* w) {
    const int lane = threadIdx.x & 31;
    const float* ml = p.ml_part + ((size_t)r * p.H + h) * p.NS * 2;
    const float m = lane < p.NS ? ml[2 * lane] : -INFINITY, l = lane < p.NS ? ml[2 * lane + 1] : 0.f;
    const float M = warp_max(m), e = m == -INFINITY ? 0.f : ex2(m - M);
    float f = 1.f / warp_sum(e * l);
    if (p.off_gate >= 0 && p.head_gate) f *= gate_sigmoid(p.proj[(size_t)r * p.ldp + p.off_gate + h]);
    w[lane] = e * f;
}
__device__ __forceinline__ float4 merged4(const LatentOut& p, int r, int h, int c, const float* w) {
    const float* op = p.o_part + ((size_t)r * p.H + h) * p.NS * p.dlp + c;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
    for (int s = 0; s < p.NS; ++s) {
        const float4 v = *reinterpret_cast<const float4*>(op + (size_t)s * p.dlp);
        a.x = fmaf(w[s], v.x, a.x); a.y = fmaf(w[s], v.y, a.y); a.z = fmaf(w[s], v.z, a.z); a.w = fmaf(w[s], v.w, a.w);
    }
    return a;
}

__global__ void __launch_bounds__(128) latent_combine_kernel(LatentOut p, bf16* __restrict__ out) {
    __shared__ float w[32];
    const int r = blockIdx.x, h = blockIdx.y;
    pdl_wait();
    pdl_launch_dependents();
    if (p.row_seq[r] < 0) return;
    if (threadIdx.x < 32) split_weights(p, r, h, w);
    __syncthreads();
    for (int c = threadIdx.x * 4; c < p.dlp; c += 512) {
        const float4 a = merged4(p, r, h, c, w);
        bf162* d = reinterpret_cast<bf162*>(out + ((size_t)r * p.H + h) * p.dlp + c);
        d[0] = __floats2bfloat162_rn(a.x, a.y); d[1] = __floats2bfloat162_rn(a.z, a.w);
    }
}

constexpr int kOutCols = 32;          // value channels per block of latent_out
template <typename T, int MT>
__global__ void __launch_bounds__(256) latent_out_kernel(LatentOut p, const T* __restrict__ w_uv, T* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) float lsm[];              // [MT][dlp]
    __shared__ float w[MT][32];
    const int h = blockIdx.y, r0 = blockIdx.z * MT, nr = min(MT, p.rows - r0), t = threadIdx.x, n0 = blockIdx.x * kOutCols, n1 = min(p.dv, n0 + kOutCols);
    prefetch_rows(w_uv + ((size_t)h * p.dv + n0) * p.dlp, (size_t)(n1 - n0) * p.dlp);
    pdl_wait();
    pdl_launch_dependents();
    if (p.NS > 1) {
        if ((t >> 5) < nr && p.row_seq[r0 + (t >> 5)] >= 0) split_weights(p, r0 + (t >> 5), h, w[t >> 5]);
        __syncthreads();
        for (int i = t * 4; i < MT * p.dlp; i += 1024) {
            const int m = i / p.dlp, c = i - m * p.dlp;
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
            if (m < nr && p.row_seq[r0 + m] >= 0) a = merged4(p, r0 + m, h, c, w[m]);
            *reinterpret_cast<float4*>(lsm + i) = a;
        }
    } else {
        const T* x = reinterpret_cast<const T*>(p.o_lat) + ((size_t)r0 * p.H + h) * p.dlp;
        for (int i = t; i < MT * p.dlp; i += 256) {
            const int m = i / p.dlp, c = i - m * p.dlp;
            lsm[i] = m < nr ? act_f(x[(size_t)m * p.H * p.dlp + c]) : 0.f;
        }
    }
    __syncthreads();
    small_products<T, MT>(w_uv + (size_t)h * p.dv * p.dlp, p.dlp, n0, n1, lsm, p.dlp, [&](int n, const float (&a)[MT]) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
            if (m < nr) {
                const float g = p.off_gate >= 0 && !p.head_gate ? gate_sigmoid(p.proj[(size_t)(r0 + m) * p.ldp + p.off_gate + (size_t)h * p.dv + n]) : 1.f;
                out[(size_t)(r0 + m) * ldo + (size_t)h * p.dv + n] = to_act<T>(a[m] * g);
            }
    });
}

// x [rows, ldo] *= sigmoid(gate), column by column (the many-row form's gate per value channel)
__global__ void __launch_bounds__(256) gate_rows_kernel(bf16* __restrict__ x, int ldo, const float* __restrict__ gate, int ldg, int n) {
    const int r = blockIdx.y, i = blockIdx.x * 256 + threadIdx.x;
    pdl_wait();
    pdl_launch_dependents();
    if (i < n) x[(size_t)r * ldo + i] = __float2bfloat16(__bfloat162float(x[(size_t)r * ldo + i]) * gate_sigmoid(gate[(size_t)r * ldg + i]));
}

template <int NV, int MG>
static int launch_latent(const LatentAttn& p, int tiles, cudaStream_t st) {
    const size_t smem = LatentCfg<NV, MG>::smem(p.dlp + p.drp);
    if (smem > 226 * 1024) return -1;
    static bool attr = false;
    if (!attr) { cudaFuncSetAttribute(latent_attn_kernel<NV, MG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024); attr = true; }
    if (p.C == 1) {
        launch_pdl((latent_attn_kernel<NV, MG>), dim3(tiles, p.NS), 256, smem, st, p);
        return (int)cudaGetLastError();
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles, p.NS); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = 1; at[0].val.clusterDim.y = p.C; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = pdl_enabled_flag() ? 2 : 1;
    return (int)cudaLaunchKernelEx(&cfg, latent_attn_kernel<NV, MG>, p);
}
template <int NV>
static int launch_latent_rows(const LatentAttn& p, int mg, int tiles, cudaStream_t st) {
    return mg == 1 ? launch_latent<NV, 1>(p, tiles, st) : (mg == 2 ? launch_latent<NV, 2>(p, tiles, st) : launch_latent<NV, 4>(p, tiles, st));
}
static int row_tiles(int run_rows, int H) { return run_rows * H <= 16 ? 1 : (run_rows * H <= 32 ? 2 : 4); }
static LatentPrep latent_prep_params(const void* qsrc, int ldq, const void* proj, int ldp, int off_kv, const void* kv_norm, float eps, const void* inv_freq, const void* w_uk, void* q,
                                     void* q_nope, void* cache, const void* block_table, int max_pages, int page, const void* row_seq, const void* row_pos,
                                     int rows, int H, int dn, int dnp, int dr, int dl) {
    LatentPrep p;
    p.qsrc = (const float*)qsrc; p.ldq = ldq; p.proj = (const float*)proj; p.ldp = ldp; p.off_kv = off_kv; p.kv_norm = (const float*)kv_norm; p.eps = eps;
    p.inv_freq = (const double*)inv_freq; p.w_uk = w_uk; p.q = q; p.q_nope = (bf16*)q_nope; p.cache = cache; p.block_table = (const int*)block_table;
    p.max_pages = max_pages; p.page = page; p.row_seq = (const int*)row_seq; p.row_pos = (const int*)row_pos; p.rows = rows; p.H = H; p.dn = dn;
    p.dnp = dnp; p.dr = dr; p.drp = (dr + 15) / 16 * 16; p.dl = dl; p.dlp = (dl + 15) / 16 * 16;
    return p;
}
constexpr int kMaxSplits = 128;       // sixteen clusters' partial sums
static int cluster_of(int NS) { return NS >= 8 ? 8 : NS; }
static bool splits_ok(int NS) { return NS == 1 || NS == 2 || NS == 4 || (NS >= 8 && NS % 8 == 0 && NS <= kMaxSplits); }
// the tensor-core kernel covers latents of up to 512 channels whose tiles fit an SM's shared memory
static bool latent_tc(int dlp, int drp, int f32) { return !f32 && dlp <= 512 && dlp + drp <= 656; }

}  // namespace lsb
using namespace lsb;

// padded width of the latent and of the rotated part in cache rows and queries
LSB_API int lsb_latent_pad(int d) { return (d + 15) / 16 * 16; }

// Key splits worth having for steps of `rows` single tokens over up to `seen` keys: 1, 2, 4 or a multiple of 8.
LSB_API int lsb_latent_splits(int rows, int H, int dl, int dr, int seen, int f32) {
    if (!latent_tc((dl + 15) / 16 * 16, (dr + 15) / 16 * 16, f32)) return 1;
    const int mg = row_tiles(1, H), blocks = rows * ((H + 16 * mg - 1) / (16 * mg)), kt = mg == 4 ? 32 : 64;
    const int most = (seen + kt - 1) / kt;                        // no split shorter than a key tile
    // clusters of eight: 14 of them are resident at a time, 16 are not; 12 leave the merge less to add up (one row of 16 heads, 8192 keys, both kernels:
    // 20.8 us with 64 splits, 22.0 with 96, 22.8 with 112, 27.3 with 128; a few keys more and 64 splits have three tiles each instead of two)
    int ns = 96 / blocks < most ? 96 / blocks : most;
    if (ns >= 8) return ns / 8 * 8;
    ns = 148 / blocks < most ? 148 / blocks : most;
    return ns >= 4 ? 4 : (ns >= 2 ? 2 : 1);
}
// Partial sums per (row, head) that NS splits leave to lsb_latent_out (1: none, the attention kernel writes its result): o_part [rows, H, this, dlp].
LSB_API int lsb_latent_partials(int NS) { return NS / cluster_of(NS); }

// Queries (rows of ldq from qsrc on, heads of dn unrotated and dr rotated channels) in the latent space and the cache append.  w_uk: [H, dlp, dnp] (dn padded to dnp % 8 == 0 with zeros).  off_kv < 0: nothing is appended.
LSB_API int lsb_latent_query(const void* qsrc, int ldq, const void* proj, int ldp, int off_kv, const void* kv_norm, float eps, const void* inv_freq, const void* w_uk,
                             void* q, void* q_nope, void* cache, const void* block_table, int max_pages, int page, const void* row_seq,
                             const void* row_pos, int rows, int H, int dn, int dnp, int dr, int dl, int f32, void* err, void* stream) {
    if (rows < 1 || dnp % 8 || dnp < dn || dr % 2 || dr < 0 || dl < 1) return -1;
    const LatentPrep p = latent_prep_params(qsrc, ldq, proj, ldp, off_kv, kv_norm, eps, inv_freq, w_uk, q, q_nope, cache, block_table, max_pages, page, row_seq, row_pos,
                                            rows, H, dn, dnp, dr, dl);
    cudaStream_t st = (cudaStream_t)stream;
    if (!f32 && rows >= 8) {
        const int D = p.dlp + p.drp;
        launch_pdl((latent_prep_kernel), rows, 256, 0, st, p);
        const int rc = lsb_gemm_bf16_tc_batched(q, q_nope, w_uk, rows, p.dlp, dnp, H, H * dnp, dnp, dnp, (long long)p.dlp * dnp, H * D, D, 1, err, stream);
        return rc ? rc : (int)cudaGetLastError();
    }
    const int mt = rows >= 4 ? 4 : (rows >= 2 ? 2 : 1);
    const dim3 grid((p.dlp + kQueryCols - 1) / kQueryCols + 1, H, (rows + mt - 1) / mt);
    const size_t smem = (size_t)mt * dnp * 4;
    if (smem > 48 * 1024) return -1;
#define LSB_LQ(T, M) launch_pdl((latent_query_kernel<T, M>), grid, 256, smem, st, p)
    if (f32) { if (mt == 4) LSB_LQ(float, 4); else if (mt == 2) LSB_LQ(float, 2); else LSB_LQ(float, 1); }
    else { if (mt == 4) LSB_LQ(bf16, 4); else if (mt == 2) LSB_LQ(bf16, 2); else LSB_LQ(bf16, 1); }
#undef LSB_LQ
    LSB_CHECK_LAUNCH();
}

// A run of rows of one sequence (row_pos consecutive, T positions in all after the append) with keys and values written out per head: q [rows, H, dnw + drp];
// kv [Tm, H dnw unrotated keys | H dvp values | drp shared rotated part], read by lsb_attn_run.  w_kv: [H dnw + H dvp, dlp], padding rows and columns zero;
// lat: scratch [Tm, dlp].  base: the first position that any row sees, row 0 of lat and kv.  Tm >= T - base: rows the product runs over (those past
// T - base are never read).
LSB_API int lsb_latent_expand(const void* qsrc, int ldq, const void* proj, int ldp, int off_kv, const void* kv_norm, float eps, const void* inv_freq, const void* w_kv,
                              void* q, void* lat, void* kv, void* cache, const void* block_table, int max_pages, int page, const void* row_seq,
                              const void* row_pos, int rows, int base, int T, int Tm, int H, int dn, int dnw, int dr, int dl, int dvp, void* err, void* stream) {
    if (rows < 1 || base < 0 || T - base < rows || Tm < T - base || dnw % 16 || dnw < dn || dvp % 16 || dr % 2 || dr < 0 || dl < 1) return -1;
    const LatentPrep p = latent_prep_params(qsrc, ldq, proj, ldp, off_kv, kv_norm, eps, inv_freq, nullptr, q, nullptr, cache, block_table, max_pages, page, row_seq, row_pos,
                                            rows, H, dn, dnw, dr, dl);
    cudaStream_t st = (cudaStream_t)stream;
    const int N = H * (dnw + dvp), ldkv = N + p.drp;
    launch_pdl((latent_rows_kernel), rows, 256, 0, st, p, dnw);
    launch_pdl((latent_gather_kernel), (T - base + 3) / 4, 128, 0, st, (const bf16*)cache, (const int*)block_table, max_pages, page, (const int*)row_seq, base, T, p.dlp, p.drp,
               (bf16*)lat, (bf16*)kv, ldkv, N);
    const int rc = lsb_gemm_bf16_tc(kv, lat, w_kv, nullptr, Tm, N, p.dlp, p.dlp, p.dlp, ldkv, 1, nullptr, 0, err, nullptr, stream);
    return rc ? rc : (int)cudaGetLastError();
}

// Attention of the step's rows.  NS: key splits (lsb_latent_splits; runs of rows use 1).  One partial sum: o_lat [rows, H, dlp], gated; more: o_part /
// ml_part, merged by lsb_latent_out.  seq_row0 / seq_nrows: the step's sequences (consecutive positions each); run_rows: the largest number of rows one of them has.
// window: sliding window (0: none); off_gate: one gate per head (-1: none, or none before lsb_latent_out).
LSB_API int lsb_latent_attn(const void* q, const void* cache, const void* block_table, int max_pages, int page, const void* row_seq, const void* row_pos,
                            const void* seq_row0, const void* seq_nrows, int nseq, int run_rows, const void* proj, int ldp, int off_gate, void* o_lat,
                            void* o_part, void* ml_part, int NS, int rows, int H, int dl, int dr, int window, float scale, int f32, void* stream) {
    if (rows < 1 || !splits_ok(NS) || (lsb_latent_partials(NS) > 1 && (!o_part || !ml_part)) || dl < 1 || dr < 0 || window < 0) return -1;
    const int dlp = lsb_latent_pad(dl), drp = lsb_latent_pad(dr), D = dlp + drp;
    cudaStream_t st = (cudaStream_t)stream;
    if (latent_tc(dlp, drp, f32)) {
        LatentAttn p;
        p.q = (const bf16*)q; p.cache = (const bf16*)cache; p.block_table = (const int*)block_table; p.max_pages = max_pages; p.page = page;
        p.row_seq = (const int*)row_seq; p.row_pos = (const int*)row_pos; p.seq_row0 = (const int*)seq_row0; p.seq_nrows = (const int*)seq_nrows;
        p.nseq = nseq; p.run_rows = run_rows; p.proj = (const float*)proj; p.ldp = ldp; p.off_gate = off_gate; p.out = (bf16*)o_lat;
        p.o_part = (float*)o_part; p.ml_part = (float*)ml_part; p.H = H; p.dlp = dlp; p.drp = drp; p.window = window; p.NS = NS; p.C = cluster_of(NS); p.scale2 = scale * kLog2e;
        const int mg = row_tiles(run_rows, H), bm = 16 * mg;
        const long long tiles = run_rows == 1 ? (long long)rows * ((H + bm - 1) / bm) : (long long)rows * H / bm + nseq;
        if (tiles > 0x7fffffff) return -1;
        const int nv = dlp <= 64 ? 1 : (dlp <= 128 ? 2 : (dlp <= 256 ? 4 : 8));
        if (nv == 1) return launch_latent_rows<1>(p, mg, (int)tiles, st);
        if (nv == 2) return launch_latent_rows<2>(p, mg, (int)tiles, st);
        if (nv == 4) return launch_latent_rows<4>(p, mg, (int)tiles, st);
        return launch_latent_rows<8>(p, mg, (int)tiles, st);
    }
    if (NS != 1) return -1;
    AttnParams p;
    p.q = q; p.cache = cache; p.block_table = (const int*)block_table; p.max_pages = max_pages; p.page = page; p.row_seq = (const int*)row_seq;
    p.row_pos = (const int*)row_pos; p.proj = (const float*)proj; p.ldp = ldp; p.off_gate = off_gate; p.head_gate = 1; p.ldc = p.dkh = D; p.off_v = p.off_ks = 0;
    p.out = o_lat; p.ldo = H * dlp; p.o_part = p.ml_part = nullptr; p.rows = rows; p.H = H; p.G = 1; p.dk = p.dkp = D; p.dv = p.dvp = dlp; p.NS = 1;
    p.window = window; p.scale = scale; p.slope = nullptr;
    const size_t smem = (size_t)(D + 256 + dlp) * 4;
    if (smem > 48 * 1024) return -1;
    if (f32) launch_pdl((attn_exact_kernel<float>), dim3(rows, H), 128, smem, st, p);
    else launch_pdl((attn_exact_kernel<bf16>), dim3(rows, H), 128, smem, st, p);
    LSB_CHECK_LAUNCH();
}

// Value up-projection: out [rows, ldo] = W_uv o_lat, heads side by side; NS (partial sums) > 1: o_lat is first made from them (and gated).
// w_uv: [H, dv, dlp].  off_gate: one gate per head (head_gate; applied here when NS > 1 only, otherwise the attention kernel has done it) or per value
// channel (of the result), -1: none.
LSB_API int lsb_latent_out(void* out, int ldo, void* o_lat, const void* o_part, const void* ml_part, int NS, const void* w_uv, const void* proj, int ldp,
                           int off_gate, int head_gate, const void* row_seq, int rows, int H, int dl, int dv, int f32, void* err, void* stream) {
    if (rows < 1 || NS < 1 || NS > 32 || (NS > 1 && (!o_part || !ml_part || f32)) || dl < 1 || dv < 1) return -1;
    const int dlp = lsb_latent_pad(dl);
    cudaStream_t st = (cudaStream_t)stream;
    LatentOut o{o_lat, (const float*)o_part, (const float*)ml_part, NS, (const float*)proj, ldp, off_gate, head_gate, (const int*)row_seq, rows, H, dlp, dv};
    if (!f32 && rows >= 8) {
        if (NS > 1) launch_pdl((latent_combine_kernel), dim3(rows, H), 128, 0, st, o, (bf16*)o_lat);
        if (dv % 8 == 0 && ldo % 8 == 0) {
            const int rc = lsb_gemm_bf16_tc_batched(out, o_lat, w_uv, rows, dv, dlp, H, H * dlp, dlp, dlp, (long long)dv * dlp, ldo, dv, 1, err, stream);
            if (rc) return rc;
            if (off_gate >= 0 && !head_gate)
                launch_pdl((gate_rows_kernel), dim3((H * dv + 255) / 256, rows), 256, 0, st, (bf16*)out, ldo, (const float*)proj + off_gate, ldp, H * dv);
            return (int)cudaGetLastError();
        }
        o.NS = 1;
    }
    const int mt = rows >= 4 ? 4 : (rows >= 2 ? 2 : 1);
    const dim3 grid((dv + kOutCols - 1) / kOutCols, H, (rows + mt - 1) / mt);
    const size_t smem = (size_t)mt * dlp * 4;
    if (smem > 47 * 1024) return -1;
#define LSB_LO(T, M) launch_pdl((latent_out_kernel<T, M>), grid, 256, smem, st, o, (const T*)w_uv, (T*)out, ldo)
    if (f32) { if (mt == 4) LSB_LO(float, 4); else if (mt == 2) LSB_LO(float, 2); else LSB_LO(float, 1); }
    else { if (mt == 4) LSB_LO(bf16, 4); else if (mt == 2) LSB_LO(bf16, 2); else LSB_LO(bf16, 1); }
#undef LSB_LO
    LSB_CHECK_LAUNCH();
}

LSB_API int lsb_trace_set_latent(void* buf) { return lsb_trace_install(buf); }
