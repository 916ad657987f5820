// Windowed grouped-query attention: heads / kv_heads query heads share a key/value head, rotary positions, queries and
// keys divided by their root mean square after the rotation, soft-capped scores, a sliding window.
//
// Per layer a slot holds two rings of `cap` positions, K (kv_heads, cap, dimp) and V (kv_heads, cap, vdp); position p lives
// in row p % cap.  cap covers the window and one prefill call (or every position), and is a multiple of 64.
//
// The rotation pairs component i with i + dims/2; the rows of the query and key matrices are packed with the two members
// of a pair next to each other.  A dot product and a root mean square do not care about the order of a head's components.
//
//   decode, short portions   k_grouped_attn: a cluster of CTAs per (query row, kv head) splits the visible keys; the 16
//                            rows of an MMA tile are the query heads of the group.  In a decode step (OWN) the kernel also
//                            rotates and norms the row's queries and its new key, and appends key and value.
//   prefill                  k_qk_rows rotates, norms and appends; k_grouped_prefill walks query tile x key tile.
//   32-bit                   k_grouped_attn_f32 after k_qk_rows.
//
// Scores, caps, softmax and weights are 32-bit; a bf16 MMA takes a weight as hi + lo bf16 pairs (latent_attn.cuh).
#pragma once
#include "latent_attn.cuh"

namespace vuib {

constexpr int GA_MAX_DIM = 256;    // padded query/key and value sizes of a head

__device__ __forceinline__ int ring_row(int p, int cap) { return p % cap; }

// limit * tanh(s / limit); 0: no cap
__device__ __forceinline__ float soft_cap(float s, float limit) { return limit > 0.f ? limit * tanhf(s / limit) : s; }
// The same through one exponential, with an absolute error of a few 2^-24 * limit.
__device__ __forceinline__ float soft_cap_fast(float s, float limit, float two_over) {
    if (!(limit > 0.f)) return s;
    const float e = __expf(fminf(fabsf(s) * two_over, 80.f));     // exp(2 |s| / limit)
    return copysignf(limit - __fdividef(2.f * limit, e + 1.f), s);
}

struct QkHead {        // what a head's components go through after the projection
    const float2* trig;   // (max_seq, rot_dims / 2) (cos, sin)
    int dim, dimp, rot_dims;
    float eps;
    int norm;             // divide by the root mean square
};

// One warp: a projected head, pairs in adjacent columns, in P float2 per lane; rotated and normed in place.
template <int P>
__device__ __forceinline__ void qk_load(const QkHead& a, const float* src, int lane, float2 (&v)[P]) {
#pragma unroll
    for (int j = 0; j < P; ++j) v[j] = 2 * (lane + 32 * j) < a.dimp ? __ldcg(reinterpret_cast<const float2*>(src) + lane + 32 * j) : make_float2(0.f, 0.f);
}
template <int P>
__device__ __forceinline__ void qk_turns(const QkHead& a, int pos, int lane, float2 (&cs)[P]) {
    const float2* tr = a.trig + (size_t)pos * (a.rot_dims / 2);
#pragma unroll
    for (int j = 0; j < P; ++j) cs[j] = 2 * (lane + 32 * j) < a.rot_dims ? __ldg(tr + lane + 32 * j) : make_float2(1.f, 0.f);
}
template <int P>
__device__ __forceinline__ void qk_finish(const QkHead& a, const float2 (&cs)[P], float2 (&v)[P]) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < P; ++j) {
        v[j] = rotate_pair(v[j].x, v[j].y, cs[j]);
        ss = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, ss));
    }
    if (!a.norm) return;
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
#pragma unroll
    for (int j = 0; j < P; ++j) {
        v[j].x *= r;
        v[j].y *= r;
    }
}
template <class T, int P>
__device__ __forceinline__ void qk_put(const QkHead& a, const float2 (&v)[P], T* dst, int lane) {
#pragma unroll
    for (int j = 0; j < P; ++j)
        if (2 * (lane + 32 * j) < a.dimp) Store<T>::put2(dst + 2 * (lane + 32 * j), v[j].x, v[j].y);
}

struct GroupedCache {
    void* cache;               // slots of this layer
    size_t slot_elems, off_v;  // elements of a slot; where V starts in it
    int cap, dimp, vdp;
    template <class T> __device__ __forceinline__ T* k(int slot, int g) const {
        return static_cast<T*>(cache) + (size_t)slot * slot_elems + (size_t)g * cap * dimp;
    }
    template <class T> __device__ __forceinline__ T* v(int slot, int g) const {
        return static_cast<T*>(cache) + (size_t)slot * slot_elems + off_v + (size_t)g * cap * vdp;
    }
};

struct QkRowsArgs {
    const float* raw; int ldraw;   // (M, ldraw): query heads | key heads from column n_k | value heads from column n_v
    int n_k, n_v;
    void* q;                       // (M, H, dimp) T
    GroupedCache c;
    QkHead h;
    const int32_t* row_slot;
    const int32_t* row_pos;
    int H, G;
};

// A warp takes U pieces of P * 64 columns of one row: its query heads, its key heads, then pieces of its values.
static __host__ __device__ __forceinline__ int qk_groups(int H, int G, int vdp, int P, int U) {
    return (H + G + (G * vdp + 64 * P - 1) / (64 * P) + U - 1) / U;
}

template <class T, int P, int U>
static __global__ void __launch_bounds__(LM_THREADS) k_qk_rows(QkRowsArgs a, int M) {
    pdl_trigger();
    pdl_wait();
    const int heads = a.H + a.G, n_v = a.G * a.c.vdp, groups = qk_groups(a.H, a.G, a.c.vdp, P, U);
    const int lane = threadIdx.x & 31, w = blockIdx.x * LM_WARPS + (threadIdx.x >> 5), m = w / groups, k0 = (w - m * groups) * U;
    if (m >= M) return;
    const int pos = __ldcg(a.row_pos + m), slot = __ldcg(a.row_slot + m);
    const float* src = a.raw + (size_t)m * a.ldraw;
    float2 v[U][P], cs[P];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int k = k0 + u;
        const bool head = k < heads;
        const float2* p = reinterpret_cast<const float2*>(src + (k < a.H ? k * a.c.dimp : head ? a.n_k + (k - a.H) * a.c.dimp : a.n_v + (k - heads) * 64 * P)) + lane;
        const int left = head ? a.c.dimp : n_v - (k - heads) * 64 * P;      // columns of this piece
#pragma unroll
        for (int j = 0; j < P; ++j) v[u][j] = 2 * (lane + 32 * j) < left ? __ldcg(p + 32 * j) : make_float2(0.f, 0.f);
    }
    qk_turns<P>(a.h, pos, lane, cs);
    float ss[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        ss[u] = 0.f;
#pragma unroll
        for (int j = 0; j < P; ++j) {
            if (k0 + u < heads) v[u][j] = rotate_pair(v[u][j].x, v[u][j].y, cs[j]);
            ss[u] = fmaf(v[u][j].x, v[u][j].x, fmaf(v[u][j].y, v[u][j].y, ss[u]));
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int u = 0; u < U; ++u) ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o);
    const int row = ring_row(pos, a.c.cap);
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int k = k0 + u;
        if (k < heads) {
            const float r = a.h.norm ? 1.0f / sqrtf(ss[u] / (float)a.h.dim + a.h.eps) : 1.f;
#pragma unroll
            for (int j = 0; j < P; ++j) {
                v[u][j].x *= r;
                v[u][j].y *= r;
            }
            qk_put<T, P>(a.h, v[u], k < a.H ? static_cast<T*>(a.q) + ((size_t)m * a.H + k) * a.c.dimp
                                            : a.c.k<T>(slot, k - a.H) + (size_t)row * a.c.dimp, lane);
        } else {
#pragma unroll
            for (int j = 0; j < P; ++j) {
                const int c = (k - heads) * 64 * P + 2 * (lane + 32 * j), g = c / a.c.vdp;
                if (c < n_v) Store<T>::put2(a.c.v<T>(slot, g) + (size_t)row * a.c.vdp + c - g * a.c.vdp, v[u][j].x, v[u][j].y);
            }
        }
    }
}

// ---------------------------------------------------------------------------
// One query row at a time, keys split over a cluster (bf16).
// ---------------------------------------------------------------------------
struct GroupedAttnArgs {
    QkRowsArgs r;             // OWN: rows to rotate, norm and append; q is unused
    const bf16* q;            // !OWN: (M, H, dimp)
    bf16* out; int ldo;       // (M, ldo): head h in columns h * vdp
    int window, max_seq, n_slots;
    int keys, nbuf;           // key tile, key tiles in shared memory
    int hpg, hgroups;         // query heads of a kv head, groups of 16 of them
    float scale, softcap;
    FastDiv k_vecs, v_vecs;   // dimp / 8, vdp / 8
};

static inline size_t grouped_attn_smem(int dimp, int vdp, int keys, int nbuf) {
    const size_t kv = (size_t)nbuf * keys * (dimp + 8 + vdp + 8) * 2, sums = (size_t)16 * (vdp + 4) * 4;   // share their space
    return (size_t)16 * (dimp + 8) * 2 + (kv > sums ? kv : sums) + 16 * (LA_KEYS + 4) * 4 + 2 * 16 * (LA_KEYS + 8) * 2 + 16 * 4 +
           16 * 8 + (size_t)(dimp + vdp) * 2;
}

template <int NT, bool OWN>  // n-tiles (8 value columns) per warp
static __global__ void __launch_bounds__(LM_THREADS) k_grouped_attn(GroupedAttnArgs a, int CL) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    pdl_trigger();
    const int dimp = a.r.c.dimp, vdp = a.r.c.vdp, cap = a.r.c.cap;
    const int ldk = dimp + 8, ldv = vdp + 8, lds = vdp + 4;
    constexpr int SP = LA_KEYS + 4, PP = LA_KEYS + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);
    bf16* Ks = Qs + 16 * ldk;
    bf16* Vs = Ks + (size_t)a.nbuf * a.keys * ldk;
    float* Os = reinterpret_cast<float*>(Ks);          // [16][lds], once the keys are used up
    const size_t kv_bytes = (size_t)a.nbuf * a.keys * (ldk + ldv) * 2, os_bytes = (size_t)16 * lds * 4;
    float* Ss = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(Ks) + (kv_bytes > os_bytes ? kv_bytes : os_bytes));
    bf16* Ph = reinterpret_cast<bf16*>(Ss + 16 * SP);
    bf16* Pl = Ph + 16 * PP;
    float* corr_s = reinterpret_cast<float*>(Pl + 16 * PP);
    float* ml_s = corr_s + 16;                          // [16][2]
    bf16* own_k = reinterpret_cast<bf16*>(ml_s + 32);   // the row's new key and value
    bf16* own_v = own_k + dimp;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int sp = blockIdx.x % CL, hg = blockIdx.x / CL % a.hgroups, kvh = blockIdx.x / CL / a.hgroups, m = blockIdx.y;
    const int h0 = kvh * a.hpg + hg * 16, nh = min(16, a.hpg - hg * 16);
    if (OWN) {   // the keys of this split, as the row table reads now, on their way to L2: a hint only, read again below
        const int s_ = min(max(__ldcg(a.r.row_slot + m), 0), a.n_slots - 1), p_ = min(max(__ldcg(a.r.row_pos + m), 0), a.max_seq - 1);
        const int lo = max(0, p_ + 1 - a.window) & ~(LA_UNIT - 1);
        int ups, ns;
        latent_splits(p_ + 1 - lo, LA_UNIT, CL, ups, ns);
        const int k0 = min(p_, lo + sp * ups * LA_UNIT), k1 = min(p_, min(lo + (sp + 1) * ups * LA_UNIT, k0 + 2 * LA_KEYS));
        const bf16 *kb = a.r.c.k<bf16>(s_, kvh), *vb = a.r.c.v<bf16>(s_, kvh);
        const int r0 = ring_row(k0, cap);
        for (int i = tid * 16; i < (k1 - k0) * dimp; i += LM_THREADS * 16) {
            const int e = r0 * dimp + i;
            asm volatile("prefetch.global.L2 [%0];" ::"l"(kb + (e < cap * dimp ? e : e - cap * dimp)));
        }
        for (int i = tid * 16; i < (k1 - k0) * vdp; i += LM_THREADS * 16) {
            const int e = r0 * vdp + i;
            asm volatile("prefetch.global.L2 [%0];" ::"l"(vb + (e < cap * vdp ? e : e - cap * vdp)));
        }
    }
    pdl_wait();
    const int slot = __ldcg(a.r.row_slot + m), pos = __ldcg(a.r.row_pos + m);
    const int first = max(0, pos + 1 - a.window), lo = first & ~(LA_UNIT - 1);
    int ups, ns;
    latent_splits(pos + 1 - lo, LA_UNIT, CL, ups, ns);
    const int k_begin = min(pos + 1, lo + sp * ups * LA_UNIT), k_end = min(pos + 1, lo + (sp + 1) * ups * LA_UNIT);
    const int n_tiles = (k_end - k_begin + a.keys - 1) / a.keys;     // 0 for a split without keys
    const bool owner = OWN && k_end == pos + 1 && k_begin <= pos;    // this split has the row's own key
    const bf16 *kb = a.r.c.k<bf16>(slot, kvh), *vb = a.r.c.v<bf16>(slot, kvh);
    const int nkv = dimp / 8, nvv = vdp / 8;
    const int ring0 = ring_row(k_begin, cap);
    auto wrap = [&](int r) { return r < cap ? r : r - cap; };    // a call's keys span no more than the ring
    auto fetch = [&](int tile) {
        bf16* kd = Ks + (size_t)(tile % a.nbuf) * a.keys * ldk;
        bf16* vd = Vs + (size_t)(tile % a.nbuf) * a.keys * ldv;
        const int k0 = k_begin + tile * a.keys, n = min(a.keys, k_end - k0) - (owner && tile == n_tiles - 1 ? 1 : 0);
        const int n16 = (min(a.keys, k_end - k0) + 15) / 16 * 16;    // zero rows up to the next MMA step
        const int r0 = ring0 + tile * a.keys;
        for (int i = tid; i < n16 * nkv; i += LM_THREADS) {
            const int key = a.k_vecs.div(i), v = i - key * nkv;
            const int row = wrap(r0 + key);
            cp_async16(kd + key * ldk + v * 8, kb + (size_t)(key < n ? row : 0) * dimp + v * 8, key < n);
        }
        for (int i = tid; i < n16 * nvv; i += LM_THREADS) {
            const int key = a.v_vecs.div(i), v = i - key * nvv;
            const int row = wrap(r0 + key);
            cp_async16(vd + key * ldv + v * 8, vb + (size_t)(key < n ? row : 0) * vdp + v * 8, key < n);
        }
        cp_async_commit();
    };
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};   // heads 2*warp, 2*warp + 1
    const int col0 = warp * NT * 8;
    if (n_tiles > 0) {
        if (!OWN) {
            const bf16* qb = a.q + ((size_t)m * a.r.H + h0) * dimp;
            for (int i = tid; i < 16 * nkv; i += LM_THREADS)
                cp_async16(Qs + i * 8 + a.k_vecs.div(i) * 8, qb + (i < nh * nkv ? i : 0) * 8, i < nh * nkv);
        }
        fetch(0);
        if (OWN) {
            const float* src = a.r.raw + (size_t)m * a.r.ldraw;
            const int row = ring_row(pos, cap);
            const bool store = owner && hg == 0;
            constexpr int P = GA_MAX_DIM / 64;
            float2 cs[P], v[P];
            qk_turns<P>(a.r.h, pos, lane, cs);
            for (int i = warp; i < 17; i += LM_WARPS) {
                const int q = i == LM_WARPS - 1 ? 16 : i == 16 ? LM_WARPS - 1 : i;     // the key is the last warp's first
                if (q >= nh && q < 16) {
                    for (int c = lane; c < dimp / 2; c += 32) reinterpret_cast<uint32_t*>(Qs + q * ldk)[c] = 0u;
                    continue;
                }
                if (q == 16 && !owner) continue;
                qk_load<P>(a.r.h, src + (q < 16 ? (h0 + q) * dimp : a.r.n_k + kvh * dimp), lane, v);
                qk_finish<P>(a.r.h, cs, v);
                qk_put<bf16, P>(a.r.h, v, q < 16 ? Qs + q * ldk : own_k, lane);
                if (q == 16 && store) qk_put<bf16, P>(a.r.h, v, a.r.c.k<bf16>(slot, kvh) + (size_t)row * dimp, lane);
            }
            if (owner)
                for (int c = 2 * tid; c < vdp; c += 2 * LM_THREADS) {
                    const float2 v = __ldcg(reinterpret_cast<const float2*>(src + a.r.n_v + kvh * vdp + c));
                    Store<bf16>::put2(own_v + c, v.x, v.y);
                    if (store) Store<bf16>::put2(a.r.c.v<bf16>(slot, kvh) + (size_t)row * vdp + c, v.x, v.y);
                }
        }
    }
    const int ksteps = dimp / 16;
    const float two_over = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
    for (int tile = 0; tile < n_tiles; ++tile) {
        const bool ahead = a.nbuf > 1 && tile + 1 < n_tiles;
        if (ahead) fetch(tile + 1);
        if (ahead) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        bf16* K = Ks + (size_t)(tile % a.nbuf) * a.keys * ldk;
        bf16* V = Vs + (size_t)(tile % a.nbuf) * a.keys * ldv;
        const int k0 = k_begin + tile * a.keys, left = min(a.keys, k_end - k0);   // keys of this tile in range
        if (owner && tile == n_tiles - 1) {                // uniform over the CTA
            if (tid < nkv) *reinterpret_cast<uint4*>(K + (left - 1) * ldk + tid * 8) = *reinterpret_cast<const uint4*>(own_k + tid * 8);
            else if (tid - nkv < nvv) *reinterpret_cast<uint4*>(V + (left - 1) * ldv + (tid - nkv) * 8) = *reinterpret_cast<const uint4*>(own_v + (tid - nkv) * 8);
            __syncthreads();
        }
        // ---- scores of 16 heads x 16 keys per warp
        if (warp * 16 < left) {
            float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
            const bf16* qp = Qs + ((lane & 7) + ((lane >> 3) & 1) * 8) * ldk + (lane >> 4) * 8;
            const bf16* kp = K + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 2
            for (int ks = 0; ks < ksteps; ++ks) {
                uint32_t q[4], b[4];
                ldsm_x4(q, qp + ks * 16);
                ldsm_x4(b, kp + ks * 16);      // keys +0..7 (k low, k high), keys +8..15
                mma_bf16(s0, q, b[0], b[1]);
                mma_bf16(s1, q, b[2], b[3]);
            }
            auto put = [&](int h, int k, float a0, float a1) {
                auto score = [&](int key, float s) {
                    return key < left && k0 + key >= first ? soft_cap_fast(s * a.scale, a.softcap, two_over) : NEG_BIG;
                };
                *reinterpret_cast<float2*>(Ss + h * SP + k) = make_float2(score(k, a0), score(k + 1, a1));
            };
            const int key = warp * 16 + 2 * t;
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
            uint32_t hi0, lo0, hi1, lo1;
            split_bf16x2(p0, p1, hi0, lo0);
            split_bf16x2(p2, p3, hi1, lo1);
            *reinterpret_cast<uint2*>(Ph + h * PP + 4 * lane) = make_uint2(hi0, hi1);
            *reinterpret_cast<uint2*>(Pl + h * PP + 4 * lane) = make_uint2(lo0, lo1);
            if (lane == 0) corr_s[h] = c;
        }
        __syncthreads();
        // ---- sums over the tile's values
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
            const bf16* vp = V + (j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + col0 + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                if (col0 + i * 8 < vdp) {    // uniform over the warp; vdp is a multiple of 16
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
    // ---- partial sums, maxima and totals for the cluster
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int col = col0 + i * 8 + 2 * t;
        if (col0 + i * 8 < vdp) {
            *reinterpret_cast<float2*>(Os + g * lds + col) = make_float2(acc[i][0], acc[i][1]);
            *reinterpret_cast<float2*>(Os + (g + 8) * lds + col) = make_float2(acc[i][2], acc[i][3]);
        }
    }
    if (lane == 0)
#pragma unroll
        for (int i = 0; i < 2; ++i) *reinterpret_cast<float2*>(ml_s + (2 * warp + i) * 2) = make_float2(m_run[i], l_run[i]);
    cluster_arrive();
    cluster_wait();
    // ---- merge in split order: pairs of columns of the valid heads over the cluster's threads
    for (int e = sp * LM_THREADS + tid; e < nh * vdp / 2; e += CL * LM_THREADS) {
        const int h = e / (vdp / 2), c = 2 * (e - h * (vdp / 2));
        float2 p[LA_MAX_CL], o[LA_MAX_CL];
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s) {
            p[s] = s < ns ? ld_cluster2(cluster_addr(ml_s + h * 2, s)) : make_float2(NEG_BIG, 0.f);
            o[s] = s < ns ? ld_cluster2(cluster_addr(Os + h * lds + c, s)) : make_float2(0.f, 0.f);
        }
        float mx = NEG_BIG, l = 0.f, v0 = 0.f, v1 = 0.f;
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s) mx = fmaxf(mx, p[s].x);
#pragma unroll
        for (int s = 0; s < LA_MAX_CL; ++s) {
            const float w = __expf(p[s].x - mx);
            l = fmaf(w, p[s].y, l);
            v0 = fmaf(w, o[s].x, v0);
            v1 = fmaf(w, o[s].y, v1);
        }
        const float inv = 1.0f / l;
        Store<bf16>::put2(a.out + (size_t)m * a.ldo + (size_t)(h0 + h) * vdp + c, v0 * inv, v1 * inv);
    }
    __syncwarp();
    cluster_arrive();   // a peer may still be reading this CTA's sums
    cluster_wait();
}

// ---------------------------------------------------------------------------
// Prefill: CTA = (tile of up to 64 consecutive positions of a slot, query head), keys 64 at a time (bf16).
// ---------------------------------------------------------------------------
constexpr int GP_TILE = 64;

struct GroupedPrefillArgs {
    const bf16* q;            // (M, H, dimp), rotated and normed
    GroupedCache c;
    const int4* tiles;        // 2 per tile; the first: (first row, rows, slot, first position)
    bf16* out; int ldo;
    int H, hpg, window;
    float scale, softcap;
    FastDiv key_vecs;         // 16-byte pieces of a key and its value
};

static inline size_t grouped_prefill_smem(int dimp, int vdp) { return (size_t)2 * GP_TILE * (dimp + 8 + vdp + 8) * 2; }

template <int KS, int NV>  // most 16-wide steps of a query/key head, most 16-column groups of a value
static __global__ void __launch_bounds__(128) k_grouped_prefill(GroupedPrefillArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dimp = a.c.dimp, vdp = a.c.vdp, ldk = dimp + 8, ldv = vdp + 8;
    bf16* Ks = reinterpret_cast<bf16*>(smem_raw);          // [2][64][ldk]
    bf16* Vs = Ks + (size_t)2 * GP_TILE * ldk;             // [2][64][ldv]
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, nks = dimp / 16, nvg = vdp / 16;
    const int4 ta = a.tiles[2 * blockIdx.x];
    const int row0 = ta.x, nrows = ta.y, pos0 = ta.w, n_keys = pos0 + nrows;
    const bf16 *kb = a.c.k<bf16>(ta.z, h / a.hpg), *vb = a.c.v<bf16>(ta.z, h / a.hpg);
    const int n_kv = dimp / 8, n_all = n_kv + vdp / 8;
    const int k_first = max(0, pos0 + 1 - a.window) & ~(GP_TILE - 1);
    auto fetch = [&](int k0, int buf) {       // cap is a multiple of the tile: a tile does not wrap
        bf16* kd = Ks + (size_t)buf * GP_TILE * ldk;
        bf16* vd = Vs + (size_t)buf * GP_TILE * ldv;
        const int r0 = ring_row(k0, a.c.cap);
        for (int i = tid; i < GP_TILE * n_all; i += 128) {
            const int key = a.key_vecs.div(i), v = i - key * n_all;
            const bool ok = k0 + key < n_keys;
            const size_t row = ok ? r0 + key : 0;
            if (v < n_kv) cp_async16(kd + key * ldk + v * 8, kb + row * dimp + v * 8, ok);
            else cp_async16(vd + key * ldv + (v - n_kv) * 8, vb + row * vdp + (v - n_kv) * 8, ok);
        }
        cp_async_commit();
    };
    fetch(k_first, 0);
    const int r_lo = warp * 16 + g, r_hi = r_lo + 8;
    const bool ok_lo = r_lo < nrows, ok_hi = r_hi < nrows;
    uint32_t qa[KS][4];
    {
        const bf16* q_lo = a.q + ((size_t)(row0 + (ok_lo ? r_lo : 0)) * a.H + h) * dimp;
        const bf16* q_hi = a.q + ((size_t)(row0 + (ok_hi ? r_hi : 0)) * a.H + h) * dimp;
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
    const int warp_last = pos0 + min(warp * 16 + 15, nrows - 1), warp_first = pos0 + warp * 16 + 1 - a.window;
    const bool warp_on = warp * 16 < nrows;
    const int p_lo = pos0 + r_lo, p_hi = pos0 + r_hi;
    const float two_over = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
    int buf = 0;
    for (int k0 = k_first; k0 < n_keys; k0 += GP_TILE, buf ^= 1) {
        cp_async_wait<0>();
        __syncthreads();    // this tile has landed for everyone, and everyone has left the other buffer
        if (k0 + GP_TILE < n_keys) fetch(k0 + GP_TILE, buf ^ 1);
        if (!warp_on || k0 > warp_last || k0 + GP_TILE <= warp_first) continue;   // uniform per warp
        const bf16* K = Ks + (size_t)buf * GP_TILE * ldk;
        const bf16* V = Vs + (size_t)buf * GP_TILE * ldv;
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
        float mx_lo = NEG_BIG, mx_hi = NEG_BIG;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int key = k0 + nt * 8 + 2 * t + (i & 1);
                const bool hi = i >> 1;
                const int p = hi ? p_hi : p_lo;
                const bool ok = key <= p && p - key < a.window && (hi ? ok_hi : ok_lo);
                s[nt][i] = ok ? soft_cap_fast(s[nt][i] * a.scale, a.softcap, two_over) : NEG_BIG;
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
    const float inv_lo = ok_lo ? 1.f / l_lo : 0.f, inv_hi = ok_hi ? 1.f / l_hi : 0.f;
#pragma unroll
    for (int v = 0; v < 2 * NV; ++v) {
        const int d = v * 8 + 2 * t;
        if (v * 8 < vdp) {
            bf16* dst = a.out + (size_t)h * vdp + d;
            if (ok_lo) Store<bf16>::put2(dst + (size_t)(row0 + r_lo) * a.ldo, o[v][0] * inv_lo, o[v][1] * inv_lo);
            if (ok_hi) Store<bf16>::put2(dst + (size_t)(row0 + r_hi) * a.ldo, o[v][2] * inv_hi, o[v][3] * inv_hi);
        }
    }
}

// ---------------------------------------------------------------------------
// 32 bits: CTA = (row, query head), 64 keys at a time, a warp per key for the scores, a thread per value column.
// ---------------------------------------------------------------------------
struct GroupedAttnF32Args {
    const float* q;           // (M, H, dimp)
    GroupedCache c;
    const int32_t* row_slot;
    const int32_t* row_pos;
    float* out; int ldo;
    int H, hpg, window;
    float scale, softcap;
};

static __global__ void __launch_bounds__(LM_THREADS) k_grouped_attn_f32(GroupedAttnF32Args a) {
    __shared__ __align__(16) float qs[GA_MAX_DIM];
    __shared__ float ss[64];
    pdl_trigger();
    pdl_wait();
    const int m = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dimp = a.c.dimp, vdp = a.c.vdp;
    const int slot = __ldcg(a.row_slot + m), pos = __ldcg(a.row_pos + m), first = max(0, pos + 1 - a.window);
    const float *kb = a.c.k<float>(slot, h / a.hpg), *vb = a.c.v<float>(slot, h / a.hpg);
    for (int i = tid; i < dimp; i += LM_THREADS) qs[i] = __ldcg(a.q + ((size_t)m * a.H + h) * dimp + i);
    float acc = 0.f, m_run = NEG_BIG, l_run = 0.f;    // of value column tid (GA_MAX_DIM == LM_THREADS)
    for (int k0 = first; k0 <= pos; k0 += 64) {
        const int n = min(64, pos + 1 - k0);
        __syncthreads();
        for (int j = warp; j < n; j += LM_WARPS) {
            const float* kr = kb + (size_t)ring_row(k0 + j, a.c.cap) * dimp;
            float d = 0.f;
            for (int i = 4 * lane; i < dimp; i += 128) {
                const float4 k = __ldcg(reinterpret_cast<const float4*>(kr + i)), q = *reinterpret_cast<const float4*>(qs + i);
                d = fmaf(q.x, k.x, fmaf(q.y, k.y, fmaf(q.z, k.z, fmaf(q.w, k.w, d))));
            }
            d = warp_sum(d);
            if (lane == 0) ss[j] = soft_cap(d * a.scale, a.softcap);
        }
        __syncthreads();
        float mx = m_run;
        for (int j = 0; j < n; ++j) mx = fmaxf(mx, ss[j]);
        const float c = expf(m_run - mx);
        acc *= c;
        l_run *= c;
        m_run = mx;
        for (int j = 0; j < n; ++j) {
            const float p = expf(ss[j] - mx);
            l_run += p;
            if (tid < vdp) acc = fmaf(p, __ldcg(vb + (size_t)ring_row(k0 + j, a.c.cap) * vdp + tid), acc);
        }
    }
    if (tid < vdp) a.out[(size_t)m * a.ldo + (size_t)h * vdp + tid] = acc / l_run;
}

}  // namespace vuib
