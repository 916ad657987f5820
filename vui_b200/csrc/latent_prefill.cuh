// Expanded form of latent attention for a prefill: per layer, the cached latents of the call's sequences are gathered
// into consecutive rows (k_latent_gather), one GEMM turns them into every head's keys and values, and k_latent_prefill
// walks query tile x key tile on the tensor cores as k_prefill_attn (prefill_attn.cuh) does: QK^T by mma.sync, online
// softmax with the causal bound, P V with the weights as hi + lo bf16 pairs.  The rotated key part, shared by all
// heads, is read from the cache.
//
// Key tiles start at multiples of 64 from position 0, and an expanded key depends on its position's cache row alone:
// cutting a prompt elsewhere gives the same rows.
#pragma once
#include "latent_attn.cuh"

namespace vuib {

constexpr int LP_TILE = 64;      // query rows per tile, keys per step
constexpr int LP_MAX_QK = 256, LP_MAX_V = 128;

static inline bool latent_prefill_fits(int qk, int v) { return qk <= LP_MAX_QK && v <= LP_MAX_V; }

struct LatentGatherArgs {
    const bf16* cache;       // (n_slots, max_seq, Dp)
    const int4* segs;        // n_segs of (slot, keys, first expanded row, -), first rows ascending
    int n_segs, rows;
    bf16* out;               // (rows, ldo): the c columns
    int ldo, Rp, Dp, max_seq;
};

static __global__ void __launch_bounds__(256) k_latent_gather(LatentGatherArgs a) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (r >= a.rows) return;
    int lo = 0, hi = a.n_segs - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (a.segs[mid].z <= r) lo = mid;
        else hi = mid - 1;
    }
    const int4 g = a.segs[lo];
    const uint4* src = reinterpret_cast<const uint4*>(a.cache + ((size_t)g.x * a.max_seq + (r - g.z)) * a.Dp);
    uint4* dst = reinterpret_cast<uint4*>(a.out + (size_t)r * a.ldo);
    for (int i = lane; i < a.ldo / 8; i += 32) dst[i] = i < a.Rp / 8 ? __ldcg(src + i) : make_uint4(0, 0, 0, 0);
}

struct LatentPrefillArgs {
    const bf16* q;           // (M, H, dimp + rotp), rotated
    const bf16* xkv;         // (rows, ldx): heads * dimp key columns, then heads * vdp value columns
    int ldx;
    const bf16* cache;       // for the rotated key part
    const int4* tiles;       // 2 per tile: (first row, rows, slot, first position), (first expanded row of the sequence, ...)
    const bf16* gate; int ldgate;
    bf16* out; int ldo;
    int H, dimp, rotp, vdim, vdp, Rp, Dp, max_seq;
    float scale;
    FastDiv key_vecs;        // 16-byte pieces of a key and its value
};

static inline size_t latent_prefill_smem(int qk, int v) { return (size_t)2 * LP_TILE * (qk + 8 + v + 8) * 2; }

template <int KS, int NV>  // most 16-wide steps of a query/key head, most 16-column groups of a value
static __global__ void __launch_bounds__(128) k_latent_prefill(LatentPrefillArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int hd = a.dimp + a.rotp, ldk = hd + 8, ldv = a.vdp + 8;
    bf16* Ks = reinterpret_cast<bf16*>(smem_raw);          // [2][64][ldk]
    bf16* Vs = Ks + (size_t)2 * LP_TILE * ldk;             // [2][64][ldv]
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, nks = hd / 16, nvg = a.vdp / 16;
    const int4 ta = a.tiles[2 * blockIdx.x], tb = a.tiles[2 * blockIdx.x + 1];
    const int row0 = ta.x, nrows = ta.y, pos0 = ta.w, n_keys = pos0 + nrows;
    const bf16* rot = a.cache + (size_t)ta.z * a.max_seq * a.Dp + a.Rp;
    const bf16* kx = a.xkv + (size_t)tb.x * a.ldx + (size_t)h * a.dimp;
    const bf16* vx = a.xkv + (size_t)tb.x * a.ldx + (size_t)a.H * a.dimp + (size_t)h * a.vdp;
    const int n_kv = a.dimp / 8, n_rv = a.rotp / 8, n_vv = a.vdp / 8, n_all = n_kv + n_rv + n_vv;
    auto fetch = [&](int k0, int buf) {
        bf16* kd = Ks + (size_t)buf * LP_TILE * ldk;
        bf16* vd = Vs + (size_t)buf * LP_TILE * ldv;
        for (int i = tid; i < LP_TILE * n_all; i += 128) {
            const int key = a.key_vecs.div(i), v = i - key * n_all;
            const bool ok = k0 + key < n_keys;
            const size_t p = ok ? k0 + key : 0;
            if (v < n_kv) cp_async16(kd + key * ldk + v * 8, kx + p * a.ldx + v * 8, ok);
            else if (v < n_kv + n_rv) cp_async16(kd + key * ldk + v * 8, rot + p * a.Dp + (v - n_kv) * 8, ok);
            else cp_async16(vd + key * ldv + (v - n_kv - n_rv) * 8, vx + p * a.ldx + (v - n_kv - n_rv) * 8, ok);
        }
        cp_async_commit();
    };
    fetch(0, 0);
    const int r_lo = warp * 16 + g, r_hi = r_lo + 8;
    const bool ok_lo = r_lo < nrows, ok_hi = r_hi < nrows;
    uint32_t qa[KS][4];
    {
        const bf16* q_lo = a.q + ((size_t)(row0 + (ok_lo ? r_lo : 0)) * a.H + h) * hd;
        const bf16* q_hi = a.q + ((size_t)(row0 + (ok_hi ? r_hi : 0)) * a.H + h) * hd;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const bool in = ks < nks;
            qa[ks][0] = in && ok_lo ? __ldcg(reinterpret_cast<const uint32_t*>(q_lo + ks * 16 + 2 * t)) : 0u;
            qa[ks][1] = in && ok_hi ? __ldcg(reinterpret_cast<const uint32_t*>(q_hi + ks * 16 + 2 * t)) : 0u;
            qa[ks][2] = in && ok_lo ? __ldcg(reinterpret_cast<const uint32_t*>(q_lo + ks * 16 + 8 + 2 * t)) : 0u;
            qa[ks][3] = in && ok_hi ? __ldcg(reinterpret_cast<const uint32_t*>(q_hi + ks * 16 + 8 + 2 * t)) : 0u;
        }
    }
    float m_lo = NEG_BIG, m_hi = NEG_BIG, l_lo = 0.f, l_hi = 0.f;
    float o[2 * NV][4];
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int warp_last = pos0 + min(warp * 16 + 15, nrows - 1);
    const bool warp_on = warp * 16 < nrows;
    int buf = 0;
    for (int k0 = 0; k0 < n_keys; k0 += LP_TILE, buf ^= 1) {
        cp_async_wait<0>();
        __syncthreads();    // this tile has landed for everyone, and everyone has left the other buffer
        if (k0 + LP_TILE < n_keys) fetch(k0 + LP_TILE, buf ^ 1);
        if (!warp_on || k0 > warp_last) continue;   // uniform per warp
        const bf16* K = Ks + (size_t)buf * LP_TILE * ldk;
        const bf16* V = Vs + (size_t)buf * LP_TILE * ldv;
        float s[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
        for (int kp = 0; kp < KS / 2; ++kp) {
            if (2 * kp + 1 < nks) {
#pragma unroll
                for (int nt = 0; nt < 8; ++nt) {
                    uint32_t b[4];
                    ldsm_x4(b, K + (nt * 8 + (lane & 7)) * ldk + kp * 32 + (lane >> 3) * 8);
                    mma_bf16(s[nt], qa[2 * kp], b[0], b[1]);
                    mma_bf16(s[nt], qa[2 * kp + 1], b[2], b[3]);
                }
            } else if (2 * kp < nks) {
#pragma unroll
                for (int nt = 0; nt < 8; ++nt) {
                    uint32_t b0, b1;
                    ldsm_x2(b0, b1, K + (nt * 8 + (lane & 7)) * ldk + kp * 32 + ((lane >> 3) & 1) * 8);
                    mma_bf16(s[nt], qa[2 * kp], b0, b1);
                }
            }
        }
        const int p_lo = pos0 + r_lo, p_hi = pos0 + r_hi;
        float mx_lo = NEG_BIG, mx_hi = NEG_BIG;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int key = k0 + nt * 8 + 2 * t + (i & 1);
                const bool hi = i >> 1, ok = key <= (hi ? p_hi : p_lo) && (hi ? ok_hi : ok_lo);
                s[nt][i] = ok ? s[nt][i] * a.scale : NEG_BIG;
                if (hi) mx_hi = fmaxf(mx_hi, s[nt][i]);
                else mx_lo = fmaxf(mx_lo, s[nt][i]);
            }
#pragma unroll
        for (int sh = 1; sh <= 2; sh <<= 1) {
            mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, sh));
            mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, sh));
        }
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
        const float c_lo = __expf(m_lo - mn_lo), c_hi = __expf(m_hi - mn_hi);
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const bool hi = i >> 1;
                const float p = s[nt][i] <= 0.5f * NEG_BIG ? 0.f : __expf(s[nt][i] - (hi ? mn_hi : mn_lo));
                s[nt][i] = p;
                if (hi) sum_hi += p;
                else sum_lo += p;
            }
#pragma unroll
        for (int sh = 1; sh <= 2; sh <<= 1) {
            sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, sh);
            sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, sh);
        }
        l_lo = l_lo * c_lo + sum_lo;
        l_hi = l_hi * c_hi + sum_hi;
        m_lo = mn_lo;
        m_hi = mn_hi;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) {
            o[i][0] *= c_lo; o[i][1] *= c_lo;
            o[i][2] *= c_hi; o[i][3] *= c_hi;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            uint32_t ph[4], pl[4];
            split_bf16x2(s[2 * j][0], s[2 * j][1], ph[0], pl[0]);
            split_bf16x2(s[2 * j][2], s[2 * j][3], ph[1], pl[1]);
            split_bf16x2(s[2 * j + 1][0], s[2 * j + 1][1], ph[2], pl[2]);
            split_bf16x2(s[2 * j + 1][2], s[2 * j + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                if (v < nvg) {
                    uint32_t b[4];
                    ldsm_x4_t(b, V + (j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + v * 16 + (lane >> 4) * 8);
                    mma_bf16(o[2 * v], ph, b[0], b[1]);
                    mma_bf16(o[2 * v + 1], ph, b[2], b[3]);
                    mma_bf16(o[2 * v], pl, b[0], b[1]);
                    mma_bf16(o[2 * v + 1], pl, b[2], b[3]);
                }
            }
        }
    }
    // ---- normalise, gate, store
    const float inv_lo = ok_lo ? 1.f / l_lo : 0.f, inv_hi = ok_hi ? 1.f / l_hi : 0.f;
#pragma unroll
    for (int v = 0; v < 2 * NV; ++v)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int d = v * 8 + 2 * t + (i & 1);
            const bool hi = i >> 1;
            if (d < a.vdim && (hi ? ok_hi : ok_lo)) {
                const size_t m = row0 + (hi ? r_hi : r_lo);
                const float gt = bf2f(a.gate[m * a.ldgate + h * a.vdim + d]);
                a.out[m * a.ldo + h * a.vdim + d] = f2bf(o[v][i] * (hi ? inv_hi : inv_lo) * gt);
            }
        }
}

}  // namespace vuib
