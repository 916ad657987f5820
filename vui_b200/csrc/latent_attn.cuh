// Latent attention: every head scores against, and sums, ONE cached row per position,
//   row = [c (Rp columns, zero-padded) | rotated key part (padded)],  Dp columns.
//
// Absorbed form (decode, short portions).  With the key matrix folded into the query projection at load time, a
// query head is a vector over the whole cached row, score = scale * q_h . row, and its output before the value
// matrix is sum_j p_j c_j.  The 16 rows of an MMA tile are the HEADS of one query row, so a key tile is read once
// for all of them.  k_latent_attn (bf16): a cluster of CTAs per query row splits the keys and merges through distributed
// shared memory; for a few rows it also applies the value matrix and the output gate, for more k_latent_value does.
// k_latent_attn_f32 leaves partial sums that meet in k_latent_out.
//
// Expanded form (prefill).  Keys and values of a call's sequences are expanded once per layer by a GEMM, and
// k_latent_prefill walks query tile x key tile per head, as k_prefill_attn (prefill_attn.cuh) does.
//
// Scores, softmax and weights are 32-bit.  A bf16 MMA takes a weight as the sum of two bf16 (p = hi + lo, 16
// significant bits), two MMAs per tile, so that the weights keep more than the 8 bits of the values they multiply.
#pragma once
#include "lm_kernels.cuh"

namespace vuib {

constexpr int LA_KEYS = 128;       // most keys per tile (bf16): 16 per warp; wide rows take 64 or 32
constexpr int LA_KEYS_F32 = 32;
constexpr int LA_MAX_SPLITS = 64;

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// p = hi + lo as packed bf16 pairs
__device__ __forceinline__ void split_bf16x2(float p0, float p1, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - f.x, p1 - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// n / d for the small indices of the copy loops: d's reciprocal rounded up, exact while n * d < 2^32.
struct FastDiv {
    uint32_t d, mul;
    FastDiv() = default;
    explicit FastDiv(int v) : d((uint32_t)v), mul((uint32_t)(((1ull << 32) + v - 1) / v)) {}   // v >= 2
    __device__ __forceinline__ int div(int n) const { return (int)__umulhi((uint32_t)n, mul); }
};

struct LatentAttnArgs {
    const void* q;            // (M, H, Dp) T
    const void* cache;        // (n_slots, max_seq, Dp) T of this layer
    const int32_t* row_slot;
    const int32_t* row_pos;
    int H, Rp, Dp, max_seq, n_slots;
    int keys;                 // per tile
    int nbuf;                 // key tiles in shared memory (1 or 2)
    float scale;
    FastDiv row_vecs, w_vecs; // Dp / 8, Rp / 8
    // bf16: value matrix and gate (fused), or the latent sums (M, H, Rp)
    const bf16* wuv;          // (H, vdim, Rp)
    const bf16* gate;         // (M, ldgate)
    bf16* out;                // fused: (M, ldo) gated values; else the latent sums
    int ldgate, ldo, vdim;
    // fp32: partial sums of the splits
    float* part;              // (M, S, H, Rp)
    float* ml;                // (M, S, H, 2): running maximum and sum
    int S;
    int col_blocks;           // grid.y = head groups of 16 x column blocks
};

// How the keys of a row of `len` positions are dealt to S splits in units of `keys`: units per split, splits in use.
__device__ __forceinline__ void latent_splits(int len, int keys, int S, int& ups, int& ns) {
    const int nu = (len + keys - 1) / keys;
    ups = (nu + S - 1) / S;
    ns = (nu + ups - 1) / ups;
}
constexpr int LA_UNIT = 16;       // the bf16 kernel deals whole 16-key MMA steps

constexpr int LA_MAX_CL = 8;      // CTAs (key splits) of a row's cluster

// fuse_heads: heads a CTA finishes itself (0: it does not); w_rows: rows of the value matrices it keeps
static inline size_t latent_attn_smem(int Dp, int Rp, int keys_per_tile, int nbuf, int fuse_heads = 0, int w_rows = 0) {
    const size_t keys = (size_t)nbuf * keys_per_tile * (Dp + 8) * 2, sums = (size_t)16 * (Rp + 4) * 4;   // share their space
    return (size_t)16 * (Dp + 8) * 2 + (keys > sums ? keys : sums) + 16 * (LA_KEYS + 4) * 4 + 2 * 16 * (LA_KEYS + 8) * 2 +
           16 * 4 + 16 * 8 + (size_t)fuse_heads * Rp * 2 + (size_t)w_rows * (Rp + LS_PAD) * 2;
}

// One cluster of CL CTAs per (query row, 16 heads): CTA = a split of the keys.  The CTAs leave their partial sums in
// shared memory; each then merges 16 / CL heads over the cluster in split order, and either writes the latent sums or
// (FUSE_V, few rows) multiplies them with its heads' value matrices and gates the result.
template <int NT, bool FUSE_V>  // n-tiles (8 columns of c) per warp
static __global__ void __launch_bounds__(LM_THREADS) k_latent_attn(LatentAttnArgs a, int CL) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    pdl_trigger();
    const int ld = a.Dp + 8, lds = a.Rp + 4;
    constexpr int SP = LA_KEYS + 4, PP = LA_KEYS + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);
    bf16* Ks = Qs + 16 * ld;
    float* Os = reinterpret_cast<float*>(Ks);          // [16][lds], once the keys are used up
    const size_t ks_bytes = (size_t)a.nbuf * a.keys * ld * 2, os_bytes = (size_t)16 * lds * 4;
    float* Ss = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(Ks) + (ks_bytes > os_bytes ? ks_bytes : os_bytes));
    bf16* Ph = reinterpret_cast<bf16*>(Ss + 16 * SP);
    bf16* Pl = Ph + 16 * PP;
    float* corr_s = reinterpret_cast<float*>(Pl + 16 * PP);
    float* ml_s = corr_s + 16;                          // [16][2]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int sp = blockIdx.x % CL, hg = blockIdx.x / CL, m = blockIdx.y;
    const int hpc = 16 / CL, h_loc0 = sp * hpc, h0 = hg * 16 + h_loc0;   // heads this CTA finishes
    const int n_fin = max(0, min(hpc, a.H - h0));
    bf16* ol = reinterpret_cast<bf16*>(ml_s + 32);      // [hpc][Rp] merged sums (FUSE_V)
    bf16* Ws = ol + (FUSE_V ? hpc * a.Rp : 0);          // [n_fin * vdim][Rp + LS_PAD] (FUSE_V)
    if constexpr (FUSE_V) {   // the value matrices are constants: on their way while the predecessor runs
        const bf16* p = a.wuv + (size_t)h0 * a.vdim * a.Rp;
        const int n = n_fin * a.vdim * a.Rp;            // a multiple of 16
        for (int i = tid; i < n / 8; i += LM_THREADS) cp_async16(Ws + i * 8 + a.w_vecs.div(i) * LS_PAD, p + i * 8, true);
        cp_async_commit();
        // The rows of this split, as the table reads now, on their way to L2: a hint only, read again below.
        const int s_ = min(max(__ldcg(a.row_slot + m), 0), a.n_slots - 1), l_ = min(max(__ldcg(a.row_pos + m), 0), a.max_seq - 1);
        int tps, ns;
        latent_splits(l_ + 1, LA_UNIT, CL, tps, ns);
        const bf16* kb = static_cast<const bf16*>(a.cache) + (size_t)s_ * a.max_seq * a.Dp;
        const int e0 = min(l_, sp * tps * LA_UNIT) * a.Dp, e1 = min(l_, min((sp + 1) * tps * LA_UNIT, sp * tps * LA_UNIT + 2 * LA_KEYS)) * a.Dp;
        for (int i = e0 + tid * 16; i < e1; i += LM_THREADS * 16) asm volatile("prefetch.global.L2 [%0];" ::"l"(kb + i));
    }
    pdl_wait();
    const int slot = __ldcg(a.row_slot + m), len = __ldcg(a.row_pos + m) + 1;
    int tps, ns;
    latent_splits(len, LA_UNIT, CL, tps, ns);
    const int k_begin = min(len, sp * tps * LA_UNIT), k_end = min(len, (sp + 1) * tps * LA_UNIT);
    const int n_tiles = (k_end - k_begin + a.keys - 1) / a.keys;     // 0 for a split without keys
    const int nv = a.Dp / 8, gph = (a.vdim + 15) / 16;
    // gates of value rows group q (16 rows of a head): this lane's rows g and g + 8; the first group's are asked for now
    auto gates = [&](int q, float& lo, float& hi) {
        const int h = q / gph, d = (q - h * gph) * 16 + g;
        const bf16* p = a.gate + (size_t)m * a.ldgate + (size_t)(h0 + h) * a.vdim + d;
        lo = t == 0 && q < n_fin * gph && d < a.vdim ? bf2f(p[0]) : 0.f;
        hi = t == 0 && q < n_fin * gph && d + 8 < a.vdim ? bf2f(p[8]) : 0.f;
    };
    float gate_lo = 0.f, gate_hi = 0.f;
    if constexpr (FUSE_V) gates(warp, gate_lo, gate_hi);
    const bf16* kb = static_cast<const bf16*>(a.cache) + (size_t)slot * a.max_seq * a.Dp;
    auto fetch = [&](int tile) {   // a tile's rows are consecutive in memory
        bf16* dst = Ks + (size_t)(tile % a.nbuf) * a.keys * ld;
        const int k0 = k_begin + tile * a.keys, keys = min(a.keys, k_end - k0), n = keys * nv, n16 = (keys + 15) / 16 * 16 * nv;
        const bf16* src = kb + (size_t)k0 * a.Dp;
        for (int i = tid; i < n16; i += LM_THREADS)      // zero rows up to the next MMA step
            cp_async16(dst + i * 8 + a.row_vecs.div(i) * 8, src + (i < n ? i : 0) * 8, i < n);
        cp_async_commit();
    };
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};   // heads 2*warp, 2*warp + 1
    const int col0 = warp * NT * 8;
    if (n_tiles > 0) {
        // queries: heads hg*16 .. +15 of this row (zero rows past the last head)
        const bf16* qb = static_cast<const bf16*>(a.q) + ((size_t)m * a.H + hg * 16) * a.Dp;
        const int nq = min(16, a.H - hg * 16) * nv;
        for (int i = tid; i < 16 * nv; i += LM_THREADS)
            cp_async16(Qs + i * 8 + a.row_vecs.div(i) * 8, qb + (i < nq ? i : 0) * 8, i < nq);
        fetch(0);
    }
    const int ksteps = a.Dp / 16;
    for (int tile = 0; tile < n_tiles; ++tile) {
        const bool ahead = a.nbuf > 1 && tile + 1 < n_tiles;
        if (ahead) fetch(tile + 1);
        if (ahead) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        const bf16* K = Ks + (size_t)(tile % a.nbuf) * a.keys * ld;
        // ---- scores of 16 heads x 16 keys per warp
        const int left = min(a.keys, k_end - k_begin - tile * a.keys);   // keys of this tile in range
        const int key = warp * 16 + 2 * t;
        if (warp * 16 < left) {
            float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
            const bf16* qp = Qs + ((lane & 7) + ((lane >> 3) & 1) * 8) * ld + (lane >> 4) * 8;
            const bf16* kp = K + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8;
#pragma unroll 2
            for (int ks = 0; ks < ksteps; ++ks) {
                uint32_t q[4], b[4];
                ldsm_x4(q, qp + ks * 16);
                ldsm_x4(b, kp + ks * 16);      // keys +0..7 (k low, k high), keys +8..15
                mma_bf16(s0, q, b[0], b[1]);
                mma_bf16(s1, q, b[2], b[3]);
            }
            auto put = [&](int h, int k, float a0, float a1) {
                *reinterpret_cast<float2*>(Ss + h * SP + k) = make_float2(k < left ? a0 * a.scale : NEG_BIG, k + 1 < left ? a1 * a.scale : NEG_BIG);
            };
            put(g, key, s0[0], s0[1]);
            put(g + 8, key, s0[2], s0[3]);
            put(g, key + 8, s1[0], s1[1]);
            put(g + 8, key + 8, s1[2], s1[3]);
        }
        __syncthreads();
        // ---- softmax rows 2*warp, 2*warp + 1; lane holds keys 4*lane .. 4*lane + 3
        const bool has = 4 * lane < (left + 15) / 16 * 16;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = 2 * warp + i;
            const float4 v = has ? *reinterpret_cast<const float4*>(Ss + h * SP + 4 * lane) : make_float4(NEG_BIG, NEG_BIG, NEG_BIG, NEG_BIG);
            float mx = fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w));
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m_run[i], mx);
            const float c = __expf(m_run[i] - mn);
            auto weight = [&](float x) { return x <= 0.5f * NEG_BIG ? 0.f : __expf(x - mn); };
            const float p0 = weight(v.x), p1 = weight(v.y), p2 = weight(v.z), p3 = weight(v.w);
            l_run[i] = l_run[i] * c + warp_sum((p0 + p1) + (p2 + p3));
            m_run[i] = mn;
            uint32_t h0, l0, h1, l1;
            split_bf16x2(p0, p1, h0, l0);
            split_bf16x2(p2, p3, h1, l1);
            *reinterpret_cast<uint2*>(Ph + h * PP + 4 * lane) = make_uint2(h0, h1);
            *reinterpret_cast<uint2*>(Pl + h * PP + 4 * lane) = make_uint2(l0, l1);
            if (lane == 0) corr_s[h] = c;
        }
        __syncthreads();
        // ---- sums over the tile's c rows
        const float c_lo = corr_s[g], c_hi = corr_s[g + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            acc[i][0] *= c_lo; acc[i][1] *= c_lo;
            acc[i][2] *= c_hi; acc[i][3] *= c_hi;
        }
#pragma unroll 2
        for (int j = 0; j < LA_KEYS / 16; ++j) {
            if (j * 16 >= left) break;
            uint32_t ph[4], pl[4];
            const int po = ((lane & 7) + ((lane >> 3) & 1) * 8) * PP + j * 16 + (lane >> 4) * 8;
            ldsm_x4(ph, Ph + po);
            ldsm_x4(pl, Pl + po);
            const bf16* vp = K + (j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + col0 + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                if (col0 + i * 8 < a.Rp) {   // uniform over the warp; Rp is a multiple of 16
                    uint32_t b[4];
                    ldsm_x4_t(b, vp + i * 8);
                    mma_bf16(acc[i], ph, b[0], b[1]);
                    mma_bf16(acc[i + 1], ph, b[2], b[3]);
                    mma_bf16(acc[i], pl, b[0], b[1]);
                    mma_bf16(acc[i + 1], pl, b[2], b[3]);
                }
            }
        }
        __syncthreads();   // the tile and the weights are used up
        if (!ahead && tile + 1 < n_tiles) fetch(tile + 1);
    }
    if (FUSE_V && n_tiles == 0) cp_async_wait<0>();      // the value matrices
    // ---- partial sums, maxima and totals for the cluster
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int col = col0 + i * 8 + 2 * t;
        if (col0 + i * 8 < a.Rp) {
            *reinterpret_cast<float2*>(Os + g * lds + col) = make_float2(acc[i][0], acc[i][1]);
            *reinterpret_cast<float2*>(Os + (g + 8) * lds + col) = make_float2(acc[i][2], acc[i][3]);
        }
    }
    if (lane == 0)
#pragma unroll
        for (int i = 0; i < 2; ++i) *reinterpret_cast<float2*>(ml_s + (2 * warp + i) * 2) = make_float2(m_run[i], l_run[i]);
    cluster_arrive();
    cluster_wait();
    // ---- merge: 256 / hpc threads per head
    const int tph = LM_THREADS / hpc, hl = tid / tph, c0 = tid % tph;
    if (hl < n_fin) {
        constexpr int CB = 2;      // columns requested together
        float w[LA_MAX_CL], o[CB][LA_MAX_CL], mx = NEG_BIG, l = 0.f;
        float2 p[LA_MAX_CL];
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s)
            p[s] = s < ns ? ld_cluster2(cluster_addr(ml_s + (h_loc0 + hl) * 2, s)) : make_float2(NEG_BIG, 0.f);
        auto ask = [&](int c) {
#pragma unroll
            for (int j = 0; j < CB; ++j)
#pragma unroll
                for (int s = 0; s < LA_MAX_CL; ++s)
                    o[j][s] = s < ns && c + j * tph < a.Rp ? ld_cluster(cluster_addr(Os + (h_loc0 + hl) * lds + c + j * tph, s)) : 0.f;
        };
        ask(c0);
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s) mx = fmaxf(mx, p[s].x);
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s) {
            w[s] = __expf(p[s].x - mx);
            l = fmaf(w[s], p[s].y, l);
        }
        const float inv = 1.0f / l;
        for (int c = c0; c < a.Rp; c += CB * tph) {
            if (c != c0) ask(c);
#pragma unroll
            for (int j = 0; j < CB; ++j) {
                if (c + j * tph >= a.Rp) break;
                float v = 0.f;
#pragma unroll
                for (int s = 0; s < LA_MAX_CL; ++s) v = fmaf(w[s], o[j][s], v);
                if constexpr (FUSE_V) ol[hl * a.Rp + c + j * tph] = f2bf(v * inv);
                else a.out[((size_t)m * a.H + h0 + hl) * a.Rp + c + j * tph] = f2bf(v * inv);
            }
        }
    }
    __syncwarp();
    cluster_arrive();
    if constexpr (FUSE_V) {
        __syncthreads();
        // 16 value rows of a head per warp (the M side), k in the lanes' own order as in k_lm_stream; the N side is this row
        const int blocks = (a.Rp + 31) / 32, nkb = a.Rp / 32;
        const int wst = a.Rp + LS_PAD;
        for (int q = warp; q < n_fin * gph; q += LM_WARPS) {
            const int h = q / gph, d0 = (q - h * gph) * 16;
            const int d_lo = d0 + g, d_hi = d0 + g + 8;
            const bf16* w0 = Ws + (h * a.vdim + min(d_lo, a.vdim - 1)) * wst + t * 8;
            const bf16* w1 = Ws + (h * a.vdim + min(d_hi, a.vdim - 1)) * wst + t * 8;
            const bf16* o = ol + h * a.Rp + t * 8;
            const size_t col = (size_t)(h0 + h) * a.vdim;
            float g_lo = gate_lo, g_hi = gate_hi;
            if (q != warp) gates(q, g_lo, g_hi);
            float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
            for (int b = 0; b < blocks; ++b) {
                const bool in = b < nkb || t < 2;        // lanes 2, 3 of a half block hold zeros
                const uint4 z = make_uint4(0, 0, 0, 0);
                const uint4 x0 = in ? *reinterpret_cast<const uint4*>(w0 + b * 32) : z, x1 = in ? *reinterpret_cast<const uint4*>(w1 + b * 32) : z;
                const uint4 y = in ? *reinterpret_cast<const uint4*>(o + b * 32) : z;
                const uint32_t a0[4] = {x0.x, x1.x, x0.y, x1.y}, a1[4] = {x0.z, x1.z, x0.w, x1.w};
                mma_bf16(c0, a0, y.x, y.y);
                mma_bf16(c1, a1, y.z, y.w);
            }
            if (t == 0) {                                // every column holds the same sums: column 0 is this lane's
                bf16* dst = a.out + (size_t)m * a.ldo + col;
                if (d_lo < a.vdim) dst[d_lo] = f2bf((c0[0] + c1[0]) * g_lo);
                if (d_hi < a.vdim) dst[d_hi] = f2bf((c0[2] + c1[2]) * g_hi);
            }
        }
    }
    cluster_wait();   // a peer may still have been reading this CTA's sums
}

// Many rows: out[m][h*vdim + d] = gate * sum_k W_uv[h][d][k] o[m][h][k] as one small product per head.  A warp owns 16
// value rows (the M side) and 16 activation rows (the N side); k is taken in the lanes' own order as in k_lm_stream.
constexpr int LV_TILES = 2;
struct LatentValueArgs {
    const bf16* wuv;       // (H, vdim, Rp)
    const bf16* o;         // (M, H, Rp)
    const bf16* gate; int ldgate;
    bf16* out; int ldo;
    int H, Rp, vdim, M;
};

static __global__ void __launch_bounds__(128) k_latent_value(LatentValueArgs a) {
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.x, d0 = (blockIdx.y * 4 + warp) * 16, m0 = blockIdx.z * 8 * LV_TILES;
    const int nkb = a.Rp / 32;                       // Rp is a multiple of 16: a half block may be left
    const bf16* w0 = a.wuv + ((size_t)h * a.vdim + min(d0 + g, a.vdim - 1)) * a.Rp + t * 8;
    const bf16* w1 = a.wuv + ((size_t)h * a.vdim + min(d0 + g + 8, a.vdim - 1)) * a.Rp + t * 8;
    const bf16* o[LV_TILES];
#pragma unroll
    for (int j = 0; j < LV_TILES; ++j) o[j] = a.o + ((size_t)min(m0 + j * 8 + g, a.M - 1) * a.H + h) * a.Rp + t * 8;
    float acc[LV_TILES][4];
#pragma unroll
    for (int j = 0; j < LV_TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    pdl_wait();
    if (d0 >= a.vdim) return;
    const int blocks = (a.Rp + 31) / 32;
    constexpr int U = 4;     // blocks requested together
    for (int b0 = 0; b0 < blocks; b0 += U) {
        uint4 x0[U], x1[U], y[U][LV_TILES];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int b = b0 + u;
            const bool in = b < nkb || (b < blocks && t < 2);   // lanes 2, 3 of a half block hold zeros
            x0[u] = in ? ldg_stream(w0 + b * 32) : make_uint4(0, 0, 0, 0);
            x1[u] = in ? ldg_stream(w1 + b * 32) : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int j = 0; j < LV_TILES; ++j) y[u][j] = in ? __ldcg(reinterpret_cast<const uint4*>(o[j] + b * 32)) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const uint32_t a0[4] = {x0[u].x, x1[u].x, x0[u].y, x1[u].y}, a1[4] = {x0[u].z, x1[u].z, x0[u].w, x1[u].w};
#pragma unroll
            for (int j = 0; j < LV_TILES; ++j) {
                mma_bf16(acc[j], a0, y[u][j].x, y[u][j].y);
                mma_bf16(acc[j], a1, y[u][j].z, y[u][j].w);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < LV_TILES; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = d0 + g + (c >> 1) * 8, m = m0 + j * 8 + 2 * t + (c & 1);
            if (d < a.vdim && m < a.M) {
                const size_t col = (size_t)h * a.vdim + d;
                a.out[(size_t)m * a.ldo + col] = f2bf(acc[j][c] * bf2f(a.gate[(size_t)m * a.ldgate + col]));
            }
        }
}

// The same in 32 bits: 16 heads x 32 keys per tile, plain FMA.
static inline size_t latent_attn_f32_smem(int Dp) {
    return (size_t)(16 + LA_KEYS_F32) * (Dp + 4) * 4 + 16 * (LA_KEYS_F32 + 1) * 4 + 16 * 4;
}

template <int NC>  // columns per thread; a CTA covers NC * 16 columns of c
static __global__ void __launch_bounds__(LM_THREADS) k_latent_attn_f32(LatentAttnArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    pdl_trigger();
    const int ld = a.Dp + 4;
    float* Qs = reinterpret_cast<float*>(smem_raw);
    float* Ks = Qs + 16 * ld;
    float* Ss = Ks + LA_KEYS_F32 * ld;
    float* corr_s = Ss + 16 * (LA_KEYS_F32 + 1);
    constexpr int SP = LA_KEYS_F32 + 1;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int sp = blockIdx.x, hg = blockIdx.y / a.col_blocks, cb = blockIdx.y % a.col_blocks, m = blockIdx.z;
    pdl_wait();
    const int slot = __ldcg(a.row_slot + m), len = __ldcg(a.row_pos + m) + 1;
    int tps, ns;
    latent_splits(len, LA_KEYS_F32, a.S, tps, ns);
    if (sp >= ns) return;
    const int k_begin = sp * tps * LA_KEYS_F32, k_end = min(len, (sp + 1) * tps * LA_KEYS_F32);
    const float* kb = static_cast<const float*>(a.cache) + (size_t)slot * a.max_seq * a.Dp;
    const float* qb = static_cast<const float*>(a.q) + ((size_t)m * a.H + hg * 16) * a.Dp;
    const int nv = a.Dp / 4;
    for (int i = tid; i < 16 * nv; i += LM_THREADS) {
        const int h = i / nv, v = i - h * nv;
        *reinterpret_cast<float4*>(Qs + h * ld + v * 4) =
            hg * 16 + h < a.H ? __ldcg(reinterpret_cast<const float4*>(qb + (size_t)h * a.Dp) + v) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int hh = tid >> 4, kk = tid & 15;
    float acc[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] = 0.f;
    float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};
    for (int k0 = k_begin; k0 < k_end; k0 += LA_KEYS_F32) {
        __syncthreads();
        for (int i = tid; i < LA_KEYS_F32 * nv; i += LM_THREADS) {
            const int key = i / nv, v = i - key * nv;
            *reinterpret_cast<float4*>(Ks + key * ld + v * 4) =
                k0 + key < k_end ? __ldcg(reinterpret_cast<const float4*>(kb + (size_t)(k0 + key) * a.Dp) + v)
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        __syncthreads();
        float d0 = 0.f, d1 = 0.f;
        for (int k = 0; k < a.Dp; k += 4) {
            const float4 q = *reinterpret_cast<const float4*>(Qs + hh * ld + k);
            const float4 x = *reinterpret_cast<const float4*>(Ks + kk * ld + k);
            const float4 y = *reinterpret_cast<const float4*>(Ks + (kk + 16) * ld + k);
            d0 = fmaf(q.x, x.x, fmaf(q.y, x.y, fmaf(q.z, x.z, fmaf(q.w, x.w, d0))));
            d1 = fmaf(q.x, y.x, fmaf(q.y, y.y, fmaf(q.z, y.z, fmaf(q.w, y.w, d1))));
        }
        Ss[hh * SP + kk] = k0 + kk < k_end ? d0 * a.scale : NEG_BIG;
        Ss[hh * SP + kk + 16] = k0 + kk + 16 < k_end ? d1 * a.scale : NEG_BIG;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = 2 * warp + i;
            const float v = Ss[h * SP + lane];
            float mx = v;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m_run[i], mx), c = expf(m_run[i] - mn);
            const float p = v <= 0.5f * NEG_BIG ? 0.f : expf(v - mn);
            l_run[i] = l_run[i] * c + warp_sum(p);
            m_run[i] = mn;
            Ss[h * SP + lane] = p;
            if (lane == 0) corr_s[h] = c;
        }
        __syncthreads();
        const float c = corr_s[hh];
#pragma unroll
        for (int i = 0; i < NC; ++i) acc[i] *= c;
        const float* vb = Ks + cb * NC * 16 + kk;
        for (int key = 0; key < LA_KEYS_F32; ++key) {
            const float p = Ss[hh * SP + key];
#pragma unroll
            for (int i = 0; i < NC; ++i)
                if (cb * NC * 16 + i * 16 < a.Rp) acc[i] = fmaf(p, vb[key * ld + i * 16], acc[i]);
        }
    }
    const size_t row = ((size_t)m * a.S + sp) * a.H + hg * 16;
    if (hg * 16 + hh < a.H)
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int col = cb * NC * 16 + i * 16 + kk;
            if (col < a.Rp) a.part[(row + hh) * a.Rp + col] = acc[i];
        }
    if (cb == 0 && lane == 0)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = 2 * warp + i;
            if (hg * 16 + h < a.H) *reinterpret_cast<float2*>(a.ml + (row + h) * 2) = make_float2(m_run[i], l_run[i]);
        }
}

// ---------------------------------------------------------------------------
// Merge of the splits in order, value matrix of the head, output gate:
//   out[m][h*vdim + d] = gate[m][h*vdim + d] * sum_k W_uv[h][d][k] o_h[k].
// CTA = (head, RT rows, slice of the value dimensions).
// ---------------------------------------------------------------------------
struct LatentOutArgs {
    const float* part;
    const float* ml;
    const int32_t* row_pos;
    const void* wuv;       // (H, vdim, Rp) T
    const void* gate;      // (M, ldgate) T, already through the sigmoid
    int ldgate;
    void* out;             // (M, ldo) T
    int ldo;
    int H, Rp, vdim, S, keys, M;
};

template <class T, int RT>
static __global__ void __launch_bounds__(LM_THREADS) k_latent_out(LatentOutArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* o_s = reinterpret_cast<float*>(smem_raw);   // [RT][Rp]
    __shared__ float wts[RT][LA_MAX_SPLITS];
    __shared__ int n_splits[RT];
    pdl_trigger();
    constexpr int VEC = Store<T>::VEC;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, r0 = blockIdx.y * RT, nr = min(RT, a.M - r0);
    const int d_per = (a.vdim + gridDim.z - 1) / gridDim.z, d0 = blockIdx.z * d_per, d1 = min(a.vdim, d0 + d_per);
    const T* W = static_cast<const T*>(a.wuv) + (size_t)h * a.vdim * a.Rp;
    pdl_wait();
    for (int r = warp; r < nr; r += LM_WARPS) {
        const int m = r0 + r;
        int tps, ns;
        latent_splits(__ldcg(a.row_pos + m) + 1, a.keys, a.S, tps, ns);
        float2 v[LA_MAX_SPLITS / 32];
        float mx = NEG_BIG;
#pragma unroll
        for (int u = 0; u < LA_MAX_SPLITS / 32; ++u) {
            const int s = lane + 32 * u;
            v[u] = s < ns ? __ldcg(reinterpret_cast<const float2*>(a.ml + (((size_t)m * a.S + s) * a.H + h) * 2))
                          : make_float2(NEG_BIG, 0.f);
            mx = fmaxf(mx, v[u].x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float l = 0.f;
#pragma unroll
        for (int u = 0; u < LA_MAX_SPLITS / 32; ++u) {
            v[u].x = expf(v[u].x - mx);
            l += v[u].x * v[u].y;
        }
        l = warp_sum(l);
#pragma unroll
        for (int u = 0; u < LA_MAX_SPLITS / 32; ++u)
            if (lane + 32 * u < ns) wts[r][lane + 32 * u] = v[u].x / l;
        if (lane == 0) n_splits[r] = ns;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nr * a.Rp; i += LM_THREADS) {
        const int r = i / a.Rp, k = i - r * a.Rp, ns = n_splits[r];
        const float* p = a.part + ((size_t)(r0 + r) * a.S * a.H + h) * a.Rp + k;
        const size_t st = (size_t)a.H * a.Rp;
        float o = 0.f;
        int s = 0;
        for (; s + 4 <= ns; s += 4) {
            float q[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) q[u] = __ldcg(p + (s + u) * st);
#pragma unroll
            for (int u = 0; u < 4; ++u) o = fmaf(q[u], wts[r][s + u], o);
        }
        for (; s < ns; ++s) o = fmaf(__ldcg(p + s * st), wts[r][s], o);
        o_s[i] = o;
    }
    __syncthreads();
    const int nv = a.Rp / VEC;
    for (int d = d0 + warp; d < d1; d += LM_WARPS) {
        float acc[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) acc[r] = 0.f;
        for (int v = lane; v < nv; v += 32) {
            float w[VEC];
            Store<T>::unpack(ldg_stream(W + (size_t)d * a.Rp + v * VEC), w);
#pragma unroll
            for (int r = 0; r < RT; ++r)
                if (r < nr)
#pragma unroll
                    for (int j = 0; j < VEC; ++j) acc[r] = fmaf(w[j], o_s[r * a.Rp + v * VEC + j], acc[r]);
        }
#pragma unroll
        for (int r = 0; r < RT; ++r) acc[r] = warp_sum(acc[r]);
        if (lane < nr) {
            const size_t c = (size_t)h * a.vdim + d;
            const float gt = Store<T>::ld(static_cast<const T*>(a.gate) + (size_t)(r0 + lane) * a.ldgate + c);
            Store<T>::put(static_cast<T*>(a.out) + (size_t)(r0 + lane) * a.ldo + c, pick<RT>(acc, lane) * gt);
        }
    }
}

}  // namespace vuib
