// Latent attention: every head scores against, and sums, ONE cached row per position,
//   row = [c (Rp columns, zero-padded) | rotated key part (padded)],  Dp columns.
//
// Absorbed form (decode, short portions).  With the key matrix folded into the query projection at load time, a
// query head is a vector over the whole cached row, score = scale * q_h . row, and its output before the value
// matrix is sum_j p_j c_j.  The 16 rows of an MMA tile are the HEADS of one query row, so a key tile is read once
// for all of them.  k_latent_attn: CTA = (split of the keys, 16 heads x a block of columns, query row); the partial
// sums meet in k_latent_out, which also applies the value matrix and the output gate.
//
// Expanded form (prefill).  Keys and values of a call's sequences are expanded once per layer by a GEMM, and
// k_latent_prefill walks query tile x key tile per head, as k_prefill_attn (prefill_attn.cuh) does.
//
// Scores, softmax and weights are 32-bit.  A bf16 MMA takes a weight as the sum of two bf16 (p = hi + lo, 16
// significant bits), two MMAs per tile, so that the weights keep more than the 8 bits of the values they multiply.
#pragma once
#include "lm_kernels.cuh"

namespace vuib {

constexpr int LA_KEYS = 64;        // keys per tile (bf16)
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

struct LatentAttnArgs {
    const void* q;            // (M, H, Dp) T
    const void* cache;        // (n_slots, max_seq, Dp) T of this layer
    const int32_t* row_slot;
    const int32_t* row_pos;
    float* part;              // (M, S, H, Rp)
    float* ml;                // (M, S, H, 2): running maximum and sum
    int H, Rp, Dp, max_seq, S;
    int col_blocks;           // grid.y = head groups of 16 x column blocks
    int nbuf;                 // key tiles in shared memory (1 or 2)
    float scale;
};

// How the keys of a row of `len` positions are dealt to S splits in tiles of `keys`: tiles per split, splits in use.
__device__ __forceinline__ void latent_splits(int len, int keys, int S, int& tps, int& ns) {
    const int nt = (len + keys - 1) / keys;
    tps = (nt + S - 1) / S;
    ns = (nt + tps - 1) / tps;
}

static inline size_t latent_attn_smem(int Dp, int nbuf) {
    return (size_t)(16 + nbuf * LA_KEYS) * (Dp + 8) * 2 + 16 * (LA_KEYS + 4) * 4 + 2 * 16 * (LA_KEYS + 8) * 2 + 16 * 4;
}

template <int NT>  // n-tiles (8 columns) per warp; a CTA covers NT * 64 columns of c
static __global__ void __launch_bounds__(LM_THREADS) k_latent_attn(LatentAttnArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    pdl_trigger();
    const int ld = a.Dp + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);
    bf16* Ks = Qs + 16 * ld;
    float* Ss = reinterpret_cast<float*>(Ks + (size_t)a.nbuf * LA_KEYS * ld);
    bf16* Ph = reinterpret_cast<bf16*>(Ss + 16 * (LA_KEYS + 4));
    bf16* Pl = Ph + 16 * (LA_KEYS + 8);
    float* corr_s = reinterpret_cast<float*>(Pl + 16 * (LA_KEYS + 8));
    constexpr int SP = LA_KEYS + 4, PP = LA_KEYS + 8;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int sp = blockIdx.x, hg = blockIdx.y / a.col_blocks, cb = blockIdx.y % a.col_blocks, m = blockIdx.z;
    pdl_wait();
    const int slot = __ldcg(a.row_slot + m), len = __ldcg(a.row_pos + m) + 1;
    int tps, ns;
    latent_splits(len, LA_KEYS, a.S, tps, ns);
    if (sp >= ns) return;
    const int k_begin = sp * tps * LA_KEYS, k_end = min(len, (sp + 1) * tps * LA_KEYS);
    const int n_tiles = (k_end - k_begin + LA_KEYS - 1) / LA_KEYS;
    const int nv = a.Dp / 8;
    const bf16* kb = static_cast<const bf16*>(a.cache) + (size_t)slot * a.max_seq * a.Dp;
    auto fetch = [&](int tile) {
        bf16* dst = Ks + (size_t)(tile % a.nbuf) * LA_KEYS * ld;
        const int k0 = k_begin + tile * LA_KEYS;
        for (int i = tid; i < LA_KEYS * nv; i += LM_THREADS) {
            const int key = i / nv, v = i - key * nv;
            const bool ok = k0 + key < k_end;
            cp_async16(dst + key * ld + v * 8, kb + (size_t)(ok ? k0 + key : k_begin) * a.Dp + v * 8, ok);
        }
        cp_async_commit();
    };
    {   // queries: heads hg*16 .. +15 of this row (zero rows past the last head)
        const bf16* qb = static_cast<const bf16*>(a.q) + ((size_t)m * a.H + hg * 16) * a.Dp;
        for (int i = tid; i < 16 * nv; i += LM_THREADS) {
            const int h = i / nv, v = i - h * nv;
            const bool ok = hg * 16 + h < a.H;
            cp_async16(Qs + h * ld + v * 8, qb + (ok ? (size_t)h * a.Dp + v * 8 : 0), ok);
        }
    }
    fetch(0);
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};   // heads 2*warp, 2*warp + 1
    const int col0 = cb * NT * 64 + warp * NT * 8;
    const int ksteps = a.Dp / 16;
    for (int tile = 0; tile < n_tiles; ++tile) {
        const bool ahead = a.nbuf > 1 && tile + 1 < n_tiles;
        if (ahead) fetch(tile + 1);
        if (ahead) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        const bf16* K = Ks + (size_t)(tile % a.nbuf) * LA_KEYS * ld;
        // ---- scores of 16 heads x 8 keys per warp, two independent accumulators
        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
        const bf16* qp = Qs + ((lane & 7) + ((lane >> 3) & 1) * 8) * ld + (lane >> 4) * 8;
        const bf16* kp = K + (warp * 8 + (lane & 7)) * ld + (lane >> 3) * 8;
        int ks = 0;
        for (; ks + 2 <= ksteps; ks += 2) {
            uint32_t a0[4], a1[4], b[4];
            ldsm_x4(a0, qp + ks * 16);
            ldsm_x4(a1, qp + ks * 16 + 16);
            ldsm_x4(b, kp + ks * 16);
            mma_bf16(s0, a0, b[0], b[1]);
            mma_bf16(s1, a1, b[2], b[3]);
        }
        if (ks < ksteps) {
            uint32_t a0[4], b0, b1;
            ldsm_x4(a0, qp + ks * 16);
            ldsm_x2(b0, b1, K + (warp * 8 + (lane & 7)) * ld + ks * 16 + ((lane >> 3) & 1) * 8);
            mma_bf16(s0, a0, b0, b1);
        }
        const int key = warp * 8 + 2 * t, left = k_end - k_begin - tile * LA_KEYS;   // keys of this tile in range
        Ss[g * SP + key] = key < left ? (s0[0] + s1[0]) * a.scale : NEG_BIG;
        Ss[g * SP + key + 1] = key + 1 < left ? (s0[1] + s1[1]) * a.scale : NEG_BIG;
        Ss[(g + 8) * SP + key] = key < left ? (s0[2] + s1[2]) * a.scale : NEG_BIG;
        Ss[(g + 8) * SP + key + 1] = key + 1 < left ? (s0[3] + s1[3]) * a.scale : NEG_BIG;
        __syncthreads();
        // ---- softmax rows 2*warp, 2*warp + 1; lane holds keys 2*lane, 2*lane + 1
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = 2 * warp + i;
            const float2 v = *reinterpret_cast<const float2*>(Ss + h * SP + 2 * lane);
            float mx = fmaxf(v.x, v.y);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m_run[i], mx);
            const float c = __expf(m_run[i] - mn);
            const float p0 = v.x <= 0.5f * NEG_BIG ? 0.f : __expf(v.x - mn);
            const float p1 = v.y <= 0.5f * NEG_BIG ? 0.f : __expf(v.y - mn);
            l_run[i] = l_run[i] * c + warp_sum(p0 + p1);
            m_run[i] = mn;
            uint32_t hi, lo;
            split_bf16x2(p0, p1, hi, lo);
            *reinterpret_cast<uint32_t*>(Ph + h * PP + 2 * lane) = hi;
            *reinterpret_cast<uint32_t*>(Pl + h * PP + 2 * lane) = lo;
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
#pragma unroll
        for (int j = 0; j < LA_KEYS / 16; ++j) {
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
    const size_t row = ((size_t)m * a.S + sp) * a.H + hg * 16;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int col = col0 + i * 8 + 2 * t;
        if (col0 + i * 8 < a.Rp) {
            if (hg * 16 + g < a.H) *reinterpret_cast<float2*>(a.part + (row + g) * a.Rp + col) = make_float2(acc[i][0], acc[i][1]);
            if (hg * 16 + g + 8 < a.H)
                *reinterpret_cast<float2*>(a.part + (row + g + 8) * a.Rp + col) = make_float2(acc[i][2], acc[i][3]);
        }
    }
    if (cb == 0 && lane == 0)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = 2 * warp + i;
            if (hg * 16 + h < a.H)
                *reinterpret_cast<float2*>(a.ml + (row + h) * 2) = make_float2(m_run[i], l_run[i]);
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
