// Building blocks of the token language models (lm.cu): row kernels, matrix products with pairwise epilogues,
// and the token sampler.  All are templates over the storage type T of weights, matrix operands and caches:
// bf16 (serving) or float (everything in 32 bits).  Whatever the type, the residual stream, norms, rotations,
// attention scores and weights, gates' arguments and logits are 32-bit.
//
// Sizes are run-time values: a model's layers may differ from one another.  Matrices are packed at load time with
// their K padded to a multiple of 64 and their rows to a multiple of 128 (zeros), so that any width can take the
// TMA / tcgen05 path; buffers keep the pad columns at zero.
//
// One epilogue functor serves all three matrix-product kernels - the weight-streaming GEMV of a few rows, the
// tcgen05 GEMM (tc_gemm.cuh) and the fp32 tile GEMM.  It is handed the sums of two adjacent weight rows (n, n + 1),
// n even, of one activation row m: rotations pair adjacent rows, gated activations interleave theirs.
#pragma once
#include "decode_kernels.cuh"
#include "tc_gemm.cuh"

namespace vuib {

constexpr int LM_THREADS = 256;
constexpr int LM_WARPS = LM_THREADS / 32;

template <class T> struct Store;
template <> struct Store<bf16> {
    static constexpr int VEC = 8;  // elements per 16-byte load
    static __device__ __forceinline__ float ld(const bf16* p) { return bf2f(*p); }
    static __device__ __forceinline__ void put(bf16* p, float v) { *p = f2bf(v); }
    static __device__ __forceinline__ void put2(bf16* p, float a, float b) {
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
    }
    static __device__ __forceinline__ void unpack(const uint4& u, float (&f)[8]) { unpack8(u, f); }
    static __device__ __forceinline__ void ld4(const bf16* p, float (&f)[4]) {
        const uint2 u = __ldcg(reinterpret_cast<const uint2*>(p));
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    }
    static __device__ __forceinline__ void put4(bf16* p, const float4& v) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
};
template <> struct Store<float> {
    static constexpr int VEC = 4;
    static __device__ __forceinline__ float ld(const float* p) { return *p; }
    static __device__ __forceinline__ void put(float* p, float v) { *p = v; }
    static __device__ __forceinline__ void put2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
    static __device__ __forceinline__ void ld4(const float* p, float (&f)[4]) {
        const float4 v = __ldcg(reinterpret_cast<const float4*>(p));
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    }
    static __device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
    static __device__ __forceinline__ void unpack(const uint4& u, float (&f)[4]) {
        f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y);
        f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
    }
};

// Sum over the block of up to N values per thread (N <= 4); every thread gets the totals.  `red` holds N * 32 floats.
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float* red) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
    __syncthreads();  // an earlier use of `red` is over
    if (lane == 0)
#pragma unroll
        for (int i = 0; i < N; ++i) red[i * 32 + warp] = v[i];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float t = 0.f;
        for (int w = 0; w < nw; ++w) t += red[i * 32 + w];
        v[i] = t;
    }
}

// Another CTA's shared memory, and the cluster's barrier.
__device__ __forceinline__ uint32_t cluster_addr(const void* p, int rank) {
    uint32_t ra;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(smem_u32(p)), "r"(rank));
    return ra;
}
__device__ __forceinline__ float ld_cluster(uint32_t a) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
    return v;
}
__device__ __forceinline__ float2 ld_cluster2(uint32_t a) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
    return v;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// Rotation of the pair (u, v) by the angle whose (cos, sin) is cs.
__device__ __forceinline__ float2 rotate_pair(float u, float v, float2 cs) {
    return make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
}

__device__ __forceinline__ float sigmoid32(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu32(float z) { return z / (1.0f + expf(-z)); }

// ---------------------------------------------------------------------------
// Embedding rows and the per-row (slot, position) table of the call.
// ---------------------------------------------------------------------------
struct EmbedArgs {
    const int64_t* tokens;     // (M)
    const void* table;         // (vocab, width) T
    float scale;
    float* x;                  // (M, ldx)
    int width, ldx, vocab;
    // decode step: slots (M) with the position taken from seq_lens; NULL in a prefill
    const int32_t* slots;
    const int32_t* seq_lens;
    // prefill: n_segs runs of (slot, first position, rows, first row); checked by the host
    const int4* segs;
    int n_segs;
    int32_t* row_slot;
    int32_t* row_pos;
    int2* row_ext;             // rows of the same portion before and after this one
    int32_t* seq_lens_out;     // prefill: the slots' new lengths
    int n_slots, max_seq;
    int32_t* flag;
};

template <class T>
static __global__ void __launch_bounds__(128) k_lm_embed(EmbedArgs a) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    if (threadIdx.x == 0) {
        int slot, pos;
        int2 ext = make_int2(0, 0);
        if (a.slots) {
            slot = a.slots[r];
            if (slot < 0 || slot >= a.n_slots) {
                atomicOr(a.flag, FLAG_BAD_SLOT);
                slot = a.n_slots - 1;
            }
            pos = a.seq_lens[slot];
            if (pos < 0 || pos >= a.max_seq) {
                atomicOr(a.flag, FLAG_BAD_POS);
                pos = pos < 0 ? 0 : a.max_seq - 1;
            }
        } else {
            int s = 0;
            while (s + 1 < a.n_segs && a.segs[s + 1].w <= r) ++s;
            const int4 g = a.segs[s];
            slot = g.x;
            pos = g.y + (r - g.w);
            ext = make_int2(r - g.w, g.w + g.z - 1 - r);
            if (r == g.w + g.z - 1) a.seq_lens_out[slot] = pos + 1;
        }
        a.row_slot[r] = slot;
        a.row_pos[r] = pos;
        a.row_ext[r] = ext;
    }
    long long tok = a.tokens[r];
    if (tok < 0 || tok >= a.vocab) {
        if (threadIdx.x == 0) atomicOr(a.flag, FLAG_BAD_CODE);
        tok = 0;
    }
    const T* src = static_cast<const T*>(a.table) + (size_t)tok * a.width;
    for (int k = threadIdx.x; k < a.width; k += blockDim.x) a.x[(size_t)r * a.ldx + k] = Store<T>::ld(src + k) * a.scale;
}

// ---------------------------------------------------------------------------
// Norm of the fp32 residual with one or two (weight, bias) pairs: a block that reads the same row through two norms
// needs its statistics once.  CENTER: layer norm, variance as the mean of the squared deviations (two passes);
// otherwise RMS norm.  A bias may be NULL.
// ---------------------------------------------------------------------------
struct NormVec {
    const float* w;
    const float* b;
};

template <class T, bool CENTER>
static __global__ void __launch_bounds__(128) k_norm_rows(const float* __restrict__ x, int ldx, int width, float eps, NormVec n1,
                                                          T* __restrict__ out1, NormVec n2, T* __restrict__ out2, int ldo,
                                                          const int32_t* __restrict__ rows, const int32_t* __restrict__ row_slot,
                                                          const int32_t* __restrict__ seq_inc, int32_t* __restrict__ seq_lens) {
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[r] : r) * ldx;
    constexpr int KEEP = 16;      // the row stays in registers up to 128 * 16 elements
    float v[KEEP];
    float s[1] = {0.f}, mean = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int k = threadIdx.x + i * 128;
        v[i] = k < width ? __ldcg(xr + k) : 0.f;
        if (CENTER) s[0] += v[i];
    }
    if (CENTER) {
        for (int k = threadIdx.x + KEEP * 128; k < width; k += 128) s[0] += __ldcg(xr + k);
        block_sums<1>(s, red);
        mean = s[0] / (float)width;
        s[0] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const float d = threadIdx.x + i * 128 < width ? v[i] - mean : 0.f;
        s[0] = fmaf(d, d, s[0]);
    }
    for (int k = threadIdx.x + KEEP * 128; k < width; k += 128) {
        const float d = __ldcg(xr + k) - mean;
        s[0] = fmaf(d, d, s[0]);
    }
    block_sums<1>(s, red);
    const float rstd = 1.0f / sqrtf(s[0] / (float)width + eps);
    auto put = [&](int k, float d) {
        Store<T>::put(out1 + (size_t)r * ldo + k, fmaf(d * rstd, __ldg(n1.w + k), n1.b ? __ldg(n1.b + k) : 0.f));
        if (out2) Store<T>::put(out2 + (size_t)r * ldo + k, fmaf(d * rstd, __ldg(n2.w + k), n2.b ? __ldg(n2.b + k) : 0.f));
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int k = threadIdx.x + i * 128;
        if (k < width) put(k, v[i] - mean);
    }
    for (int k = threadIdx.x + KEEP * 128; k < width; k += 128) put(k, __ldcg(xr + k) - mean);
    if (seq_lens && threadIdx.x == 0) {   // end of a decode step: the slots grow
        const int inc = seq_inc ? seq_inc[r] : 1;
        if (inc) seq_lens[row_slot[r]] += inc;
    }
}

// ---------------------------------------------------------------------------
// Latent attention, per position: from the fp32 projections of one row to what the cache holds,
// [RMSNorm(c) (Rp, zero-padded) | rotated key part (padded)], T.  One warp per call.
// ---------------------------------------------------------------------------
struct LatentRow {
    const float* dkv;      // (M, Dp): [c | rotated part] as the packed projection writes it
    const float* norm_w;   // (R)
    float eps;
    int R, Rp, rot, rot_dims, Dp;
    const float2* trig;    // (max_seq, rot_dims / 2) (cos, sin)
    void* cache;           // (n_slots, max_seq, Dp) T of this layer
    const int32_t* row_slot;
    const int32_t* row_pos;
    int max_seq;
};

template <class T>
__device__ __forceinline__ void latent_row(const LatentRow& a, int m, int lane) {
    constexpr int KEEP = 8;       // elements of a lane held in registers, all requested together
    const float* src = a.dkv + (size_t)m * a.Dp;
    const int slot = __ldcg(a.row_slot + m), pos = __ldcg(a.row_pos + m);
    float v[KEEP], w[KEEP], ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int k = lane + 32 * i;
        v[i] = k < a.R ? __ldcg(src + k) : 0.f;
        w[i] = k < a.R ? __ldg(a.norm_w + k) : 0.f;
    }
    const bool one = lane * 2 + 1 < a.rot;    // the first 64 rotated components
    float2 rv = one ? __ldcg(reinterpret_cast<const float2*>(src + a.Rp) + lane) : make_float2(0.f, 0.f);
    T* dst = static_cast<T*>(a.cache) + ((size_t)slot * a.max_seq + pos) * a.Dp;
    const float2* tr = a.trig + (size_t)pos * (a.rot_dims / 2);
    const float2 cs = 2 * lane < a.rot_dims ? __ldg(tr + lane) : make_float2(1.f, 0.f);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) ss = fmaf(v[i], v[i], ss);
    for (int k = lane + 32 * KEEP; k < a.R; k += 32) {
        const float u = __ldcg(src + k);
        ss = fmaf(u, u, ss);
    }
    ss = warp_sum(ss);
    const float rinv = 1.0f / sqrtf(ss / (float)a.R + a.eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (lane + 32 * i < a.R) Store<T>::put(dst + lane + 32 * i, v[i] * rinv * w[i]);
    for (int k = lane + 32 * KEEP; k < a.R; k += 32) Store<T>::put(dst + k, __ldcg(src + k) * rinv * __ldg(a.norm_w + k));
    if (one) {
        rv = rotate_pair(rv.x, rv.y, cs);
        Store<T>::put2(dst + a.Rp + 2 * lane, rv.x, rv.y);
    } else if (lane * 2 < a.rot) {            // an odd component at the end is never rotated
        Store<T>::put(dst + a.Rp + 2 * lane, __ldcg(src + a.Rp + 2 * lane));
    }
    for (int i = lane + 32; 2 * i < a.rot; i += 32) {
        float u = __ldcg(src + a.Rp + 2 * i);
        const bool pair = 2 * i + 1 < a.rot;
        float x = pair ? __ldcg(src + a.Rp + 2 * i + 1) : 0.f;
        if (2 * i < a.rot_dims) {
            const float2 o = rotate_pair(u, x, __ldg(tr + i));
            u = o.x;
            x = o.y;
        }
        Store<T>::put(dst + a.Rp + 2 * i, u);
        if (pair) Store<T>::put(dst + a.Rp + 2 * i + 1, x);
    }
}

// Many rows: cq = RMSNorm(dq) and the cache row, one CTA per row (warps 0-2: queries' latent, warp 3: cache row).
template <class T>
static __global__ void __launch_bounds__(128) k_latent_rows(LatentRow a, const float* __restrict__ dq, int lddq, int q_rank,
                                                            const float* __restrict__ q_norm, T* __restrict__ cq, int ldcq) {
    __shared__ float red[4];
    pdl_trigger();
    pdl_wait();
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* src = dq + (size_t)m * lddq;
    if (warp == 3) {
        latent_row<T>(a, m, lane);
    } else {
        float ss = 0.f;
        for (int k = threadIdx.x; k < q_rank; k += 96) {
            const float v = __ldcg(src + k);
            ss = fmaf(v, v, ss);
        }
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        bar_named(1, 96);
        const float rinv = 1.0f / sqrtf((red[0] + red[1] + red[2]) / (float)q_rank + a.eps);
        for (int k = threadIdx.x; k < ldcq; k += 96)
            Store<T>::put(cq + (size_t)m * ldcq + k, k < q_rank ? __ldcg(src + k) * rinv * __ldg(q_norm + k) : 0.f);
    }
}

// ---------------------------------------------------------------------------
// Pairwise epilogues: store(m, n, v0, v1) for the sums of weight rows n, n + 1 (n even) and activation row m.
// ---------------------------------------------------------------------------

// What an epilogue needs from global memory besides the sums may be asked for early, in two dependent steps around the
// staging: ask(m), then pre(asked, n), then store(m, n, v0, v1, pre).
struct NoEpPre {};
template <class Epi, class = void>
struct EpPre {
    typedef NoEpPre type;
    static __device__ __forceinline__ int ask(const Epi&, int) { return 0; }
    static __device__ __forceinline__ type pre(const Epi&, int, int) { return NoEpPre{}; }
    static __device__ __forceinline__ void store(const Epi& ep, int m, int n, float v0, float v1, const type&) { ep.store(m, n, v0, v1); }
};

// Everything a parallel block reads from x: [dq | dkv | gate] of the mixer, then the MLP's (gate, up) pairs.
template <class T>
struct EpBlockIn {
    int n_dq, n_kv, n_gate;   // region ends: dq rows [0, n_dq), dkv rows [n_dq, n_kv), gate rows [n_kv, n_gate)
    int n_mlp;                // first MLP row; unit u has rows n_mlp + 2u (gate), n_mlp + 2u + 1 (up)
    int ff;
    float* dq; int lddq;
    float* dkv; int lddkv;
    T* gate; int ldgate;      // sigmoid of the mixer's output gate
    T* act; int ldact;        // MLP activations
    float limit, slope, shift;
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const {
        if (n < n_dq) {
            *reinterpret_cast<float2*>(dq + (size_t)m * lddq + n) = make_float2(v0, v1);
        } else if (n < n_kv) {
            *reinterpret_cast<float2*>(dkv + (size_t)m * lddkv + (n - n_dq)) = make_float2(v0, v1);
        } else if (n < n_gate) {
            Store<T>::put2(gate + (size_t)m * ldgate + (n - n_kv), sigmoid32(v0), sigmoid32(v1));
        } else if (n >= n_mlp) {
            const int u = (n - n_mlp) >> 1;
            if (u < ff) {
                const float g = fminf(v0, limit), up = fminf(fmaxf(v1, -limit), limit);
                Store<T>::put(act + (size_t)m * ldact + u, g * sigmoid32(slope * g) * (up + shift));
            }
        }
    }
};

// Queries, head by head [plain part (n0) | rotated part], rotated at the row's position.
template <class T>
struct EpRotatedQ {
    T* q; int N, head_rows, n0, rot_dims;
    const float2* trig;
    const int32_t* row_pos;
    __device__ __forceinline__ void put(int m, int n, int j, float v0, float v1, const float2* tr) const {
        if (j >= 0 && j < rot_dims) {
            const float2 o = rotate_pair(v0, v1, tr[j >> 1]);
            v0 = o.x;
            v1 = o.y;
        }
        Store<T>::put2(q + (size_t)m * N + n, v0, v1);
    }
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const {
        if (n >= N) return;
        const int j = n % head_rows - n0;
        put(m, n, j, v0, v1, j >= 0 && j < rot_dims ? trig + (size_t)__ldcg(row_pos + m) * (rot_dims / 2) : nullptr);
    }
    __device__ __forceinline__ float2 turn(int pos, int n) const {
        const int j = n % head_rows - n0;
        return n < N && j >= 0 && j < rot_dims ? __ldg(trig + (size_t)pos * (rot_dims / 2) + (j >> 1)) : make_float2(1.f, 0.f);
    }
    // tcgen05 form: the rows' (cos, sin) are fetched while the MMAs run, TC_EPI_BYTES_PER_M of them per row
    static constexpr int STAGE_DIMS = TC_EPI_BYTES_PER_M / 4;
    __device__ __forceinline__ void stage(unsigned char* es, int m_off, int M, int tid) const {
        if (rot_dims > STAGE_DIMS) return;
        const int half = rot_dims / 2;
        float2* dst = reinterpret_cast<float2*>(es);
        for (int m = tid; m < M; m += TC_THREADS) {
            const float2* src = trig + (size_t)__ldcg(row_pos + m_off + m) * half;
            for (int i = 0; i < half; ++i) dst[m * half + i] = __ldg(src + i);
        }
    }
    __host__ __device__ size_t stage_bytes_per_row() const { return rot_dims <= STAGE_DIMS ? (size_t)rot_dims * 4 : 0; }
    __device__ __forceinline__ void store_staged(int m_off, int m, int n, float v0, float v1, const unsigned char* es) const {
        if (rot_dims > STAGE_DIMS) return store(m_off + m, n, v0, v1);
        if (n < N) put(m_off + m, n, n % head_rows - n0, v0, v1, reinterpret_cast<const float2*>(es) + m * (rot_dims / 2));
    }
};

template <class T>
struct EpPre<EpRotatedQ<T>> {
    typedef float2 type;
    static __device__ __forceinline__ int ask(const EpRotatedQ<T>& ep, int m) { return __ldcg(ep.row_pos + m); }
    static __device__ __forceinline__ float2 pre(const EpRotatedQ<T>& ep, int asked, int n) { return ep.turn(asked, n); }
    static __device__ __forceinline__ void store(const EpRotatedQ<T>& ep, int m, int n, float v0, float v1, const float2& cs) {
        if (n >= ep.N) return;
        const float2 o = rotate_pair(v0, v1, cs);   // (1, 0) turns nothing
        Store<T>::put2(ep.q + (size_t)m * ep.N + n, o.x, o.y);
    }
};

// Everything a block with one norm reads from x: the mixer's fp32 rows [0, n_raw) (a bias may be added), its gate rows
// [n_raw, n_gate) through silu, then the MLP's units through the square of relu.
template <class T>
struct EpMixIn {
    int n_raw, n_gate, n_mlp, ff;
    const float* bias;        // (n_raw) or NULL
    float* raw; int ldraw;
    T* gate; int ldgate;
    T* act; int ldact;        // columns up to a multiple of 64
    __device__ __forceinline__ void put(int m, int n, float v0, float v1, float2 b) const {
        if (n < n_raw) {
            *reinterpret_cast<float2*>(raw + (size_t)m * ldraw + n) = make_float2(v0 + b.x, v1 + b.y);
        } else if (n < n_gate) {
            Store<T>::put2(gate + (size_t)m * ldgate + (n - n_raw), silu32(v0), silu32(v1));
        } else if (n >= n_mlp && n - n_mlp < ff) {
            const float r0 = fmaxf(v0, 0.f), r1 = fmaxf(v1, 0.f);
            Store<T>::put2(act + (size_t)m * ldact + (n - n_mlp), r0 * r0, r1 * r1);
        }
    }
    __device__ __forceinline__ float2 bias_at(int n) const {
        return bias && n < n_raw ? __ldg(reinterpret_cast<const float2*>(bias + n)) : make_float2(0.f, 0.f);
    }
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const { put(m, n, v0, v1, bias_at(n)); }
};

template <class T>
struct EpPre<EpMixIn<T>> {
    typedef float2 type;
    static __device__ __forceinline__ int ask(const EpMixIn<T>&, int) { return 0; }
    static __device__ __forceinline__ float2 pre(const EpMixIn<T>& ep, int, int n) { return ep.bias_at(n); }
    static __device__ __forceinline__ void store(const EpMixIn<T>& ep, int m, int n, float v0, float v1, const float2& b) { ep.put(m, n, v0, v1, b); }
};

// x += W a in 32 bits.  Every element is added to once per launch, so the reductions have no order to depend on; they
// return nothing, so no thread waits for the old value.
struct EpAddResidual {
    float* x; int ldx, N;
    const float* bias;        // (N up to even) or NULL
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const {
        float* p = x + (size_t)m * ldx + n;
        if (bias && n < N) {
            const float2 b = __ldg(reinterpret_cast<const float2*>(bias + n));
            v0 += b.x;
            v1 += b.y;
        }
        if (n + 1 < N) asm volatile("red.global.add.v2.f32 [%0], {%1, %2};" ::"l"(p), "f"(v0), "f"(v1) : "memory");
        else if (n < N) atomicAdd(p, v0);
    }
};

// fp32 rows times a constant (logits).
struct EpLogitsF32 {
    float* out; int N;
    float scale;
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const {
        float* p = out + (size_t)m * N + n;
        if (n < N) p[0] = v0 * scale;
        if (n + 1 < N) p[1] = v1 * scale;
    }
};

// Plain T rows with a row stride (expanded keys and values of a prefill).
template <class T>
struct EpRows {
    T* out; int N, ldo;
    __device__ __forceinline__ void store(int m, int n, float v0, float v1) const {
        if (n < N) Store<T>::put2(out + (size_t)m * ldo + n, v0, v1);
    }
};

// The functor under k_gemm_tc: a thread owns weight row n and 8 activation rows; it trades halves with the thread of
// row n ^ 1, so that the even row's thread stores rows m0..m0+3 and the odd row's thread m0+4..m0+7 of the pair.
template <class F>
struct TcPair {
    F f;
    int m_off = 0;
    static constexpr bool PAIRED = false;
    static constexpr bool STAGED = false;
    __host__ __device__ TcPair shifted(int m) const { return TcPair{f, m_off + m}; }
    __device__ __forceinline__ void apply(int n, int m0, int M, const float (&v)[8], float*, const unsigned char*) const {
        const bool odd = n & 1;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float give = odd ? v[j] : v[4 + j];
            const float got = __shfl_xor_sync(0xffffffffu, give, 1);
            const int m = m0 + j + (odd ? 4 : 0);
            if (m < M) f.store(m_off + m, n & ~1, odd ? got : v[j], odd ? v[4 + j] : got);
        }
    }
};

// The same for a functor that fetches something per activation row while the MMAs run.
template <class F>
struct TcPairStaged {
    F f;
    int m_off = 0;
    static constexpr bool PAIRED = false;
    static constexpr bool STAGED = true;
    __host__ __device__ TcPairStaged shifted(int m) const { return TcPairStaged{f, m_off + m}; }
    size_t stage_bytes_per_row() const { return f.stage_bytes_per_row(); }
    __device__ __forceinline__ void stage(unsigned char* es, int, int M, int tid) const { f.stage(es, m_off, M, tid); }
    __device__ __forceinline__ void apply(int n, int m0, int M, const float (&v)[8], float*, const unsigned char* es) const {
        const bool odd = n & 1;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float give = odd ? v[j] : v[4 + j];
            const float got = __shfl_xor_sync(0xffffffffu, give, 1);
            const int m = m0 + j + (odd ? 4 : 0);
            if (m < M) f.store_staged(m_off, m, n & ~1, odd ? got : v[j], odd ? v[4 + j] : got, es);
        }
    }
};
template <class F> struct TcForm { typedef TcPair<F> type; };
template <class T> struct TcForm<EpRotatedQ<T>> { typedef TcPairStaged<EpRotatedQ<T>> type; };

// ---------------------------------------------------------------------------
// Weight-streaming products for a few rows.  Stage functors fill X tiles [RT][K] of T in shared memory and say which
// tile a weight row multiplies.  Weights are requested before the dependency wait.
//
//  k_lm_stream (bf16, up to 8 rows): a warp owns 16 weight rows (the M side of mma.sync m16n8k16) and the activation
//  rows are its N side.  A dot product does not care about the order of k, so a lane takes 8 consecutive k of its rows
//  with one 16-byte load and feeds them to the two MMAs of a 32-k block; the activations are read with the same
//  permutation.  kw warps of a CTA and ck CTAs of a cluster split K; their sums meet in shared memory in order.
//
//  k_lm_gemv (fp32, any row count in tiles of RT): a warp owns two adjacent weight rows, wk warps may split K.
// ---------------------------------------------------------------------------
constexpr int LS_PAD = 32;   // elements between X rows beyond K: eight lanes of a 16-byte read hit eight bank groups

// Two layer norms of the residual row (rows of W below `split` multiply the first).
template <class T>
struct StageLayerNorm2 {
    const float* x; int ldx, width;
    float eps;
    NormVec n1, n2;
    int split;
    const int32_t* rows;      // optional gather of x's rows
    static __host__ __device__ size_t smem(int RT, int K) { return (size_t)RT * K * (2 * sizeof(T) + 4); }
    template <int RT>
    __device__ __forceinline__ void stage(unsigned char* sm, float* red, int K, int r0, int nr) const {
        T* X1 = reinterpret_cast<T*>(sm);
        T* X2 = X1 + (size_t)RT * K;
        float* xf = reinterpret_cast<float*>(X2 + (size_t)RT * K);
        float s[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            s[r] = 0.f;
            if (r < nr) {
                const float* xr = x + (size_t)(rows ? rows[r0 + r] : r0 + r) * ldx;
                for (int k = threadIdx.x; k < width; k += LM_THREADS) {
                    const float v = __ldcg(xr + k);
                    xf[r * K + k] = v;
                    s[r] += v;
                }
            }
        }
        block_sums<RT>(s, red);
        float mean[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            mean[r] = s[r] / (float)width;
            s[r] = 0.f;
            if (r < nr)
                for (int k = threadIdx.x; k < width; k += LM_THREADS) {
                    const float d = xf[r * K + k] - mean[r];
                    s[r] = fmaf(d, d, s[r]);
                }
        }
        block_sums<RT>(s, red);
        for (int k = threadIdx.x; k < K; k += LM_THREADS) {
            const bool in = k < width;
            const float w1 = in ? __ldg(n1.w + k) : 0.f, b1 = in ? __ldg(n1.b + k) : 0.f;
            const float w2 = in && n2.w ? __ldg(n2.w + k) : 0.f, b2 = in && n2.w ? __ldg(n2.b + k) : 0.f;
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                const float d = in && r < nr ? (xf[r * K + k] - mean[r]) * (1.0f / sqrtf(s[r] / (float)width + eps)) : 0.f;
                Store<T>::put(X1 + r * K + k, fmaf(d, w1, b1));
                Store<T>::put(X2 + r * K + k, fmaf(d, w2, b2));
            }
        }
    }
    template <int RT>
    __device__ __forceinline__ const T* tile(const unsigned char* sm, int K, int n) const {
        return reinterpret_cast<const T*>(sm) + (n >= split ? (size_t)RT * K : 0);
    }
    __device__ __forceinline__ void extra(int) const {}
    static constexpr bool HAS_EXTRA = false;

    // k_lm_stream form: 8 / RT warps per row.  The norms' vectors are constants and come to shared memory before the
    // dependency wait; the row is kept there in 32 bits between the passes.
    static constexpr int TILES = 2;
    static constexpr bool K_PARTS = false;
    static __host__ __device__ size_t scratch(int RT, int K) { return (size_t)(RT + 4) * K * 4; }
    __device__ __forceinline__ void constants(float* sc, int K) const {
        const float* src[4] = {n1.w, n1.b, n2.w, n2.b};
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (src[i])
                for (int k = threadIdx.x; k < width; k += LM_THREADS) sc[i * K + k] = __ldg(src[i] + k);
    }
    template <int RT>
    __device__ __forceinline__ void stage_rows(bf16* X, int ld, float* red, float* sc, int K, int M, int) const {
        constexpr int WPR = LM_WARPS / RT, TPR = 32 * WPR, U = 4;
        const int r = threadIdx.x / TPR, i0 = threadIdx.x % TPR, warp = threadIdx.x >> 5;
        const bool on = r < M;
        const float* xr = x + (size_t)(on ? (rows ? rows[r] : r) : 0) * ldx;
        float* xs = sc + (size_t)(4 + r) * K;
        const int nv = K / 4;              // K = ldx, and the row's pad is zero
        float sum = 0.f;
        for (int q0 = i0; q0 < nv; q0 += U * TPR) {
            float4 v[U];
#pragma unroll
            for (int u = 0; u < U; ++u)
                v[u] = q0 + u * TPR < nv ? __ldcg(reinterpret_cast<const float4*>(xr) + q0 + u * TPR) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int u = 0; u < U; ++u)
                if (q0 + u * TPR < nv) {
                    reinterpret_cast<float4*>(xs)[q0 + u * TPR] = v[u];
                    sum += (v[u].x + v[u].y) + (v[u].z + v[u].w);
                }
        }
        auto row_total = [&](float t, float* buf) {
            t = warp_sum(t);
            if (WPR > 1) {
                if ((threadIdx.x & 31) == 0) buf[warp] = t;
                __syncthreads();
                t = 0.f;
#pragma unroll
                for (int w = 0; w < WPR; ++w) t += buf[r * WPR + w];
            }
            return t;
        };
        const float mean = row_total(sum, red) / (float)width;
        float m2 = 0.f;
        for (int q = i0; q < nv; q += TPR) {
            const float4 v = reinterpret_cast<const float4*>(xs)[q];
            const float f[4] = {v.x - mean, v.y - mean, v.z - mean, v.w - mean};
#pragma unroll
            for (int j = 0; j < 4; ++j) m2 = 4 * q + j < width ? fmaf(f[j], f[j], m2) : m2;
        }
        const float rstd = 1.0f / sqrtf(row_total(m2, red + LM_WARPS) / (float)width + eps);
        if (WPR == 1) __syncthreads();     // the constants are in place
        if (!on) return;
        bf16* X1 = X + (size_t)r * ld;
        bf16* X2 = X + (size_t)(RT + r) * ld;
        for (int q = i0; q < nv; q += TPR) {
            const float4 v = reinterpret_cast<const float4*>(xs)[q];
            const float f[4] = {v.x, v.y, v.z, v.w};
            float a[4], b[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int k = 4 * q + j;
                const float d = (f[j] - mean) * rstd;
                const bool in = k < width;
                a[j] = in ? fmaf(d, sc[k], sc[K + k]) : 0.f;
                b[j] = in && n2.w ? fmaf(d, sc[2 * K + k], sc[3 * K + k]) : 0.f;
            }
            Store<bf16>::put2(X1 + 4 * q, a[0], a[1]);
            Store<bf16>::put2(X1 + 4 * q + 2, a[2], a[3]);
            Store<bf16>::put2(X2 + 4 * q, b[0], b[1]);
            Store<bf16>::put2(X2 + 4 * q + 2, b[2], b[3]);
        }
    }
    __device__ __forceinline__ int tile_of(int n) const { return n >= split ? 1 : 0; }
};

// RMS norm of an fp32 row; its padding up to a multiple of 4 may be read.
template <class T>
struct StageRms {
    const float* x; int ldx, width;
    float eps;
    const float* norm_w;
    static constexpr bool HAS_EXTRA = false;
    static __host__ __device__ size_t smem(int RT, int K) { return (size_t)RT * K * sizeof(T); }
    template <int RT>
    __device__ __forceinline__ void stage(unsigned char* sm, float* red, int K, int r0, int nr) const {
        T* X = reinterpret_cast<T*>(sm);
        float s[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            s[r] = 0.f;
            if (r < nr)
                for (int k = threadIdx.x; k < width; k += LM_THREADS) {
                    const float v = __ldcg(x + (size_t)(r0 + r) * ldx + k);
                    s[r] = fmaf(v, v, s[r]);
                }
        }
        block_sums<RT>(s, red);
        for (int k = threadIdx.x; k < K; k += LM_THREADS)
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                float o = 0.f;
                if (k < width && r < nr)
                    o = __ldcg(x + (size_t)(r0 + r) * ldx + k) * (1.0f / sqrtf(s[r] / (float)width + eps)) * __ldg(norm_w + k);
                Store<T>::put(X + r * K + k, o);
            }
    }
    template <int RT>
    __device__ __forceinline__ const T* tile(const unsigned char* sm, int, int) const { return reinterpret_cast<const T*>(sm); }
    __device__ __forceinline__ void extra(int) const {}
    static constexpr int TILES = 1;
    static constexpr bool K_PARTS = false;
    static __host__ __device__ size_t scratch(int RT, int K) { return (size_t)(RT + 1) * K * 4; }
    __device__ __forceinline__ void constants(float* sc, int K) const {
        for (int k = threadIdx.x; k < K; k += LM_THREADS) sc[k] = k < width ? __ldg(norm_w + k) : 0.f;
    }
    template <int RT>
    __device__ __forceinline__ void stage_rows(bf16* X, int ld, float* red, float* sc, int K, int M, int) const {
        constexpr int WPR = LM_WARPS / RT, TPR = 32 * WPR, U = 4;
        const int r = threadIdx.x / TPR, i0 = threadIdx.x % TPR, warp = threadIdx.x >> 5;
        const bool on = r < M;
        const float* src = x + (size_t)(on ? r : 0) * ldx;
        float* xs = sc + (size_t)(1 + r) * K;
        const int nv = (width + 3) / 4;
        float ss = 0.f;
        for (int q0 = i0; q0 < K / 4; q0 += U * TPR) {
            float4 v[U];
#pragma unroll
            for (int u = 0; u < U; ++u)
                v[u] = q0 + u * TPR < nv ? __ldcg(reinterpret_cast<const float4*>(src) + q0 + u * TPR) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int q = q0 + u * TPR;
                if (q < K / 4) {
                    if (4 * q + 1 >= width) v[u].y = 0.f;     // what lies beyond the row is not part of it
                    if (4 * q + 2 >= width) v[u].z = 0.f;
                    if (4 * q + 3 >= width) v[u].w = 0.f;
                    reinterpret_cast<float4*>(xs)[q] = v[u];
                    ss = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, ss))));
                }
            }
        }
        ss = warp_sum(ss);
        if ((threadIdx.x & 31) == 0) red[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < WPR; ++w) ss += red[r * WPR + w];
        if (!on) return;
        const float rinv = 1.0f / sqrtf(ss / (float)width + eps);
        for (int q = i0; q < K / 4; q += TPR) {
            const float4 v = reinterpret_cast<const float4*>(xs)[q], w = reinterpret_cast<const float4*>(sc)[q];
            Store<bf16>::put2(X + (size_t)r * ld + 4 * q, v.x * rinv * w.x, v.y * rinv * w.y);
            Store<bf16>::put2(X + (size_t)r * ld + 4 * q + 2, v.z * rinv * w.z, v.w * rinv * w.w);
        }
    }
    __device__ __forceinline__ int tile_of(int) const { return 0; }
};

// The same of the queries' latent; the grid's last CTA appends the call's cache rows.
template <class T>
struct StageLatentQ : StageRms<T> {
    LatentRow lat;
    static constexpr bool HAS_EXTRA = true;
    __device__ __forceinline__ void extra(int M) const {
        for (int m = threadIdx.x >> 5; m < M; m += LM_WARPS) latent_row<T>(lat, m, threadIdx.x & 31);
    }
};

template <class T>
struct StageRowsT {
    const T* x; int ldx;
    static constexpr bool HAS_EXTRA = false;
    static __host__ __device__ size_t smem(int RT, int K) { return (size_t)RT * K * sizeof(T); }
    template <int RT>
    __device__ __forceinline__ void stage(unsigned char* sm, float*, int K, int r0, int nr) const {
        const int nv = K / Store<T>::VEC;
        uint4* dst = reinterpret_cast<uint4*>(sm);
        for (int i = threadIdx.x; i < nr * nv; i += LM_THREADS) {
            const int r = i / nv, v = i - r * nv;
            dst[i] = __ldcg(reinterpret_cast<const uint4*>(x + (size_t)(r0 + r) * ldx) + v);
        }
    }
    template <int RT>
    __device__ __forceinline__ const T* tile(const unsigned char* sm, int, int) const { return reinterpret_cast<const T*>(sm); }
    __device__ __forceinline__ void extra(int) const {}
    static constexpr int TILES = 1;
    static constexpr bool K_PARTS = true;   // may stage one CTA's part of K alone
    static __host__ __device__ size_t scratch(int, int) { return 0; }
    __device__ __forceinline__ void constants(float*, int) const {}
    template <int RT>
    __device__ __forceinline__ void stage_rows(bf16* X, int ld, float*, float*, int K, int M, int k0) const {
        const int nv = K / 8;
        for (int r = 0; r < M; ++r)
            for (int v = threadIdx.x; v < nv; v += LM_THREADS)
                *reinterpret_cast<uint4*>(X + (size_t)r * ld + v * 8) = __ldcg(reinterpret_cast<const uint4*>(x + (size_t)r * ldx + k0) + v);
    }
    __device__ __forceinline__ int tile_of(int) const { return 0; }
};

struct StreamArgs {
    const bf16* W;
    int K, M;
    int n_groups;     // groups of 16 weight rows
    int kw;           // warps of a CTA along K; the CTA takes 8 / kw groups at a time
    int ck;           // CTAs of a cluster along K (1, 2, 4), each with a contiguous part
};

template <int RT, class Stage, class Epi>
static __global__ void __launch_bounds__(LM_THREADS, 2) k_lm_stream(Stage st, Epi ep, StreamArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float red[2 * LM_WARPS];
    __shared__ __align__(16) float part[LM_WARPS][16][8];
    __shared__ float2 sums[LM_WARPS * 8 * 8];   // of the CTA's warps: pair of rows x activation row x group
    constexpr int U = 4;       // 32-k blocks per round, two rounds in flight
    bf16* X = reinterpret_cast<bf16*>(smem_raw);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int Kc = a.K / a.ck, ld = Kc + LS_PAD;
    pdl_trigger();
    if (Stage::HAS_EXTRA && blockIdx.x == gridDim.x - 1) {
        pdl_wait();
        st.extra(a.M);
        return;
    }
    const int n_cta = (gridDim.x - (Stage::HAS_EXTRA ? 1 : 0)) / a.ck, cta = blockIdx.x / a.ck, rank = blockIdx.x % a.ck;
    const int gpc = LM_WARPS / a.kw, gi = warp / a.kw, kp = warp % a.kw, ksplit = a.kw;
    const int nkb = Kc / 32, my_kb = (nkb - kp + ksplit - 1) / ksplit;    // this warp's blocks: kp, kp + ksplit, ...
    const int rounds = ((nkb + ksplit - 1) / ksplit + U - 1) / U;            // the same for every warp
    const int sets = (a.n_groups + gpc * n_cta - 1) / (gpc * n_cta);
    uint4 w0[2][U], w1[2][U];
    // round it of set s: weight rows g and g + 8 of the group, 8 consecutive k per lane and block
    auto load = [&](int buf, int s, int it) {
        const int grp = (s * n_cta + cta) * gpc + gi;
        const bool live = grp < a.n_groups;
        const bf16* p = a.W + (size_t)((live ? grp : 0) * 16 + g) * a.K + rank * Kc + t * 8;
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int b = it * U + u;
            const bool ok = live && b < my_kb;
            const size_t o = (size_t)(kp + b * ksplit) * 32;
            w0[buf][u] = ok ? ldg_stream(p + o) : make_uint4(0, 0, 0, 0);
            w1[buf][u] = ok ? ldg_stream(p + (size_t)8 * a.K + o) : make_uint4(0, 0, 0, 0);
        }
    };
    const int total = sets * rounds;
    load(0, 0, 0);
    if (total > 1) load(1, rounds > 1 ? 0 : 1, rounds > 1 ? 1 : 0);
    {   // a few rounds more of the first set on their way to L2
        const int grp = cta * gpc + gi;
        if (grp < a.n_groups && (t & 1) == 0)     // a hint brings one 32-byte sector
            for (int b = 2 * U; b < my_kb && b < 8 * U; ++b) {
                const bf16* p = a.W + (size_t)(grp * 16 + g) * a.K + rank * Kc + (size_t)(kp + b * ksplit) * 32 + t * 8;
                asm volatile("prefetch.global.L2 [%0];" ::"l"(p));
                asm volatile("prefetch.global.L2 [%0];" ::"l"(p + (size_t)8 * a.K));
            }
    }
    float* sc = reinterpret_cast<float*>(X + (size_t)Stage::TILES * RT * ld);
    st.constants(sc, Kc);
    pdl_wait();
    // of the output this thread stores first (below)
    const int o_m = (threadIdx.x >> 3) / gpc, o_n = ((cta * gpc + (threadIdx.x >> 3) % gpc) * 16) + 2 * (threadIdx.x & 7);
    const int asked = EpPre<Epi>::ask(ep, min(o_m, a.M - 1));
    st.template stage_rows<RT>(X, ld, red, sc, Kc, a.M, rank * Kc);
    const typename EpPre<Epi>::type first_pre = EpPre<Epi>::pre(ep, asked, o_n);
    __syncthreads();
    const int xrow = min(g, a.M - 1);   // columns past the last row repeat it and are not stored
    int s = 0, it = 0;
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[0][i] = acc[1][i] = 0.f;
    auto round = [&](int buf, int i) {
        if (it == 0)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[0][c] = acc[1][c] = 0.f;
        const int grp = (s * n_cta + cta) * gpc + gi;
        const bf16* xp = X + (size_t)(Stage::TILES > 1 ? st.tile_of(grp * 16) * RT : 0) * ld + (size_t)xrow * ld + t * 8;
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int b = it * U + u;
            if (b < my_kb) {
                const uint4 x = *reinterpret_cast<const uint4*>(xp + (size_t)(kp + b * ksplit) * 32);
                const uint32_t a0[4] = {w0[buf][u].x, w1[buf][u].x, w0[buf][u].y, w1[buf][u].y};
                const uint32_t a1[4] = {w0[buf][u].z, w1[buf][u].z, w0[buf][u].w, w1[buf][u].w};
                asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                             : "+f"(acc[0][0]), "+f"(acc[0][1]), "+f"(acc[0][2]), "+f"(acc[0][3])
                             : "r"(a0[0]), "r"(a0[1]), "r"(a0[2]), "r"(a0[3]), "r"(x.x), "r"(x.y));
                asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                             : "+f"(acc[1][0]), "+f"(acc[1][1]), "+f"(acc[1][2]), "+f"(acc[1][3])
                             : "r"(a1[0]), "r"(a1[1]), "r"(a1[2]), "r"(a1[3]), "r"(x.z), "r"(x.w));
            }
        }
        // two rounds ahead
        if (i + 2 < total) {
            int s2 = s, it2 = it + 2;
            while (it2 >= rounds) { it2 -= rounds; ++s2; }
            load(buf, s2, it2);
        }
        if (++it < rounds) return;
        it = 0;
        // the set is complete: sums meet in shared memory
        *reinterpret_cast<float2*>(&part[warp][g][2 * t]) = make_float2(acc[0][0] + acc[1][0], acc[0][1] + acc[1][1]);
        *reinterpret_cast<float2*>(&part[warp][g + 8][2 * t]) = make_float2(acc[0][2] + acc[1][2], acc[0][3] + acc[1][3]);
        __syncthreads();
        // 8 pairs of rows x M rows x gpc groups: first over the CTA's warps, then over the cluster
        const int base = (s * n_cta + cta) * gpc, n_out = gpc * 8 * a.M;
        for (int o = threadIdx.x; o < n_out; o += LM_THREADS) {
            const int pr = o & 7, gm = o >> 3, q = gm % gpc, m = gm / gpc;
            float v0 = 0.f, v1 = 0.f;
#pragma unroll
            for (int w = 0; w < LM_WARPS; ++w)
                if (w < a.kw) {
                    const float* p = &part[q * a.kw + w][2 * pr][m];
                    v0 += p[0];
                    v1 += p[8];
                }
            if (a.ck > 1) sums[o] = make_float2(v0, v1);
            else if (base + q < a.n_groups) {
                const int n = (base + q) * 16 + 2 * pr;
                EpPre<Epi>::store(ep, m, n, v0, v1, s == 0 && o < LM_THREADS ? first_pre : EpPre<Epi>::pre(ep, EpPre<Epi>::ask(ep, m), n));
            }
        }
        if (a.ck > 1) {
            cluster_arrive();
            cluster_wait();
            for (int o = rank + a.ck * threadIdx.x; o < n_out; o += a.ck * LM_THREADS) {
                const int pr = o & 7, gm = o >> 3, q = gm % gpc, m = gm / gpc;
                float2 v[4];
#pragma unroll
                for (int c = 0; c < 4; ++c) v[c] = c < a.ck ? ld_cluster2(cluster_addr(&sums[o], c)) : make_float2(0.f, 0.f);
                if (base + q < a.n_groups)
                    ep.store(m, (base + q) * 16 + 2 * pr, (v[0].x + v[1].x) + (v[2].x + v[3].x), (v[0].y + v[1].y) + (v[2].y + v[3].y));
            }
            cluster_arrive();   // no CTA leaves, or writes its sums again, while a peer may still read them
            cluster_wait();
        } else if (s + 1 < sets) {
            __syncthreads();
        }
        ++s;
    };
    for (int i = 0; i < total; i += 2) {
        round(0, i);
        if (i + 1 < total) round(1, i + 1);
    }
}

template <class T, int RT, class Stage, class Epi>
static __global__ void __launch_bounds__(LM_THREADS, 2) k_lm_gemv(Stage st, Epi ep, const T* __restrict__ W, int K, int M,
                                                                  int n_pairs, int wk) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float red[4 * 32];
    __shared__ float part[LM_WARPS][2 * RT];
    constexpr int VEC = Store<T>::VEC;
    constexpr int U = 4;       // 16-byte requests per row and round
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    if (Stage::HAS_EXTRA && blockIdx.x == gridDim.x - 1) {
        pdl_wait();
        st.extra(M);
        return;
    }
    const int pair = blockIdx.x * (LM_WARPS / wk) + warp / wk, kp = warp % wk;
    const bool live = pair < n_pairs;
    const int nv = K / VEC;                           // vectors per row
    const int v0 = kp * 32 + lane, vstep = 32 * wk;   // this lane's vectors: v0, v0 + vstep, ...
    const uint4* w0 = reinterpret_cast<const uint4*>(W + (size_t)(live ? 2 * pair : 0) * K);
    const uint4* w1 = w0 + nv;
    uint4 cur[U][2];
    auto load = [&](uint4 (&d)[U][2], int i0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int v = v0 + (i0 + u) * vstep;
            const bool ok = live && v < nv;
            d[u][0] = ok ? ldg_stream(w0 + v) : make_uint4(0, 0, 0, 0);
            d[u][1] = ok ? ldg_stream(w1 + v) : make_uint4(0, 0, 0, 0);
        }
    };
    load(cur, 0);
    pdl_wait();
    const int rounds = (nv + U * vstep - 1) / (U * vstep);
    for (int r0 = 0; r0 < M; r0 += RT) {
        const int nr = min(RT, M - r0);
        if (r0) {
            __syncthreads();
            load(cur, 0);
        }
        st.template stage<RT>(smem_raw, red, K, r0, nr);
        __syncthreads();
        const T* X = st.template tile<RT>(smem_raw, K, 2 * pair);
        float acc[2][RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) acc[0][r] = acc[1][r] = 0.f;
        for (int it = 0; it < rounds; ++it) {
            uint4 nxt[U][2];
            if (it + 1 < rounds) load(nxt, (it + 1) * U);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int v = v0 + (it * U + u) * vstep;
                if (v < nv) {
                    float a[VEC], b[VEC];
                    Store<T>::unpack(cur[u][0], a);
                    Store<T>::unpack(cur[u][1], b);
#pragma unroll
                    for (int r = 0; r < RT; ++r) {
                        if (r < nr) {
                            float xv[VEC];
                            Store<T>::unpack(*reinterpret_cast<const uint4*>(X + (size_t)r * K + v * VEC), xv);
#pragma unroll
                            for (int j = 0; j < VEC; ++j) {
                                acc[0][r] = fmaf(a[j], xv[j], acc[0][r]);
                                acc[1][r] = fmaf(b[j], xv[j], acc[1][r]);
                            }
                        }
                    }
                }
            }
            if (it + 1 < rounds) {
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    cur[u][0] = nxt[u][0];
                    cur[u][1] = nxt[u][1];
                }
            }
        }
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            acc[0][r] = warp_sum(acc[0][r]);
            acc[1][r] = warp_sum(acc[1][r]);
        }
        if (wk > 1) {
            if (lane == 0)
#pragma unroll
                for (int r = 0; r < RT; ++r) {
                    part[warp][2 * r] = acc[0][r];
                    part[warp][2 * r + 1] = acc[1][r];
                }
            __syncthreads();
            if (kp == 0) {
#pragma unroll
                for (int r = 0; r < RT; ++r)
                    for (int w = 1; w < wk; ++w) {
                        acc[0][r] += part[warp + w][2 * r];
                        acc[1][r] += part[warp + w][2 * r + 1];
                    }
            }
        }
        if (live && kp == 0 && lane < nr) ep.store(r0 + lane, 2 * pair, pick<RT>(acc[0], lane), pick<RT>(acc[1], lane));
    }
}

// ---------------------------------------------------------------------------
// fp32 tile GEMM (64 x 64 x 16, plain FMA: nothing below 32 bits) for more rows than the GEMV takes.
// Weight rows from n_split on multiply the rows x_off further down in X.
// ---------------------------------------------------------------------------
template <class Epi>
static __global__ void __launch_bounds__(256) k_gemm_f32(const float* __restrict__ X, int ldx, const float* __restrict__ W,
                                                         int K, int M, int n_split, int x_off, Epi ep) {
    __shared__ __align__(16) float Xs[16][64 + 4], Ws[16][64 + 4];
    pdl_trigger();
    pdl_wait();
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    const float* Xb = X + (n0 >= n_split ? (size_t)x_off * ldx : 0);
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
        const float4 xv = m0 + lr < M ? __ldcg(reinterpret_cast<const float4*>(Xb + (size_t)(m0 + lr) * ldx + k0 + lk))
                                      : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 wv = __ldg(reinterpret_cast<const float4*>(W + (size_t)(n0 + lr) * K + k0 + lk));
        __syncthreads();
        Xs[lk][lr] = xv.x; Xs[lk + 1][lr] = xv.y; Xs[lk + 2][lr] = xv.z; Xs[lk + 3][lr] = xv.w;
        Ws[lk][lr] = wv.x; Ws[lk + 1][lr] = wv.y; Ws[lk + 2][lr] = wv.z; Ws[lk + 3][lr] = wv.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&Xs[k][ty * 4]);
            const float4 b = *reinterpret_cast<const float4*>(&Ws[k][tx * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m < M) {
            ep.store(m, n0 + tx * 4, acc[i][0], acc[i][1]);
            ep.store(m, n0 + tx * 4 + 2, acc[i][2], acc[i][3]);
        }
    }
}

// ---------------------------------------------------------------------------
// Token sampler over fp32 logits of any vocabulary: the rule of sample_row (decode_kernels.cuh) with the
// row swept in shared strides instead of held in registers - repetition penalty, greedy (first index of the
// maximum) or temperature, top-k (every entry >= the k-th value), inverse-CDF draw from Philox keyed
// (seed; slot, draw counter, 0).  The draw counter of a slot restarts when the slot is taken by a new request.
// ---------------------------------------------------------------------------
struct TokenSampleArgs {
    float* logits;             // (B, V); a penalised row is rewritten in place
    int V;
    const SamplingCtl* ctl;
    const int32_t* slots;      // (B)
    int32_t* draw_ctr;         // (n_slots)
    float* rep_counts;         // (n_slots, V)
    int32_t* rep_hist;         // (n_slots, REP_HIST_MAX)
    int32_t* rep_head;
    int32_t* rep_filled;
    int64_t* tokens_out;       // (B)
    int n_slots;
    int32_t* flag;
};

static __global__ void __launch_bounds__(SAMPLE_THREADS) k_sample_tokens(TokenSampleArgs a) {
    __shared__ float s_f[8];
    __shared__ int s_i[8];
    __shared__ uint32_t hist[256];
    __shared__ uint32_t s_prefix, s_krem;
    __shared__ int s_pick, s_lastkept;
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, V = a.V;
    int slot = __ldcg(a.slots + r);
    if (slot < 0 || slot >= a.n_slots) {
        if (tid == 0) atomicOr(a.flag, FLAG_BAD_SLOT);
        slot = slot < 0 ? 0 : a.n_slots - 1;
    }
    const SamplingCtl ctl = *a.ctl;
    float* lg = a.logits + (size_t)r * V;
    const bool pen = ctl.rep_penalty > 1.0f;
    // penalty and argmax in one sweep
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int k = tid; k < V; k += SAMPLE_THREADS) {
        float v = lg[k];
        if (pen) {
            const float c = a.rep_counts[(size_t)slot * V + k];
            if (c != 0.f) {
                const float f = powf(ctl.rep_penalty, c);
                v = v > 0.f ? v / f : v * f;
                lg[k] = v;
            }
        }
        if (v > bv) { bv = v; bi = k; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    if (lane == 0) { s_f[warp] = bv; s_i[warp] = bi; }
    __syncthreads();
    bv = s_f[0]; bi = s_i[0];
#pragma unroll
    for (int w = 1; w < 8; ++w)
        if (s_f[w] > bv || (s_f[w] == bv && s_i[w] < bi)) { bv = s_f[w]; bi = s_i[w]; }
    if (bi < 0 || bi >= V) bi = 0;   // a row of NaNs
    __syncthreads();
    int top_k = ctl.top_k_cb0;
    if (top_k >= V) top_k = 0;
    int choice = bi;
    if (top_k != 1) {
        const float T = ctl.temperature, smax = bv / T;
        uint32_t thr = 0u;
        if (top_k > 0) {   // radix select of the top_k-th largest key, 8 bits per pass
            if (tid == 0) { s_prefix = 0u; s_krem = (uint32_t)top_k; }
            for (int pass = 0; pass < 4; ++pass) {
                const int shift = 24 - 8 * pass;
                hist[tid] = 0u;
                __syncthreads();
                const uint32_t prefix = s_prefix, pmask = pass == 0 ? 0u : (0xFFFFFFFFu << (shift + 8));
                for (int k = tid; k < V; k += SAMPLE_THREADS) {
                    const uint32_t key = order_key(lg[k] / T);
                    if ((key & pmask) == prefix) atomicAdd(&hist[(key >> shift) & 255u], 1u);
                }
                __syncthreads();
                if (tid == 0) {
                    uint32_t cum = 0u, krem = s_krem;
                    for (int d = 255; d >= 0; --d) {
                        if (cum + hist[d] >= krem) {
                            s_prefix = prefix | ((uint32_t)d << shift);
                            s_krem = krem - cum;
                            break;
                        }
                        cum += hist[d];
                    }
                }
                __syncthreads();
            }
            thr = s_prefix;
        }
        // every thread owns a contiguous piece, so that the cumulative sum runs in vocabulary order
        const int per = (V + SAMPLE_THREADS - 1) / SAMPLE_THREADS, k0 = tid * per, k1 = min(V, k0 + per);
        float loc = 0.f;
        for (int k = k0; k < k1; ++k) {
            const float sc = lg[k] / T;
            if (top_k == 0 || order_key(sc) >= thr) loc += expf(sc - smax);
        }
        float inc = loc;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float t = __shfl_up_sync(0xffffffffu, inc, o);
            if (lane >= o) inc += t;
        }
        if (lane == 31) s_f[warp] = inc;
        if (tid == 0) { s_pick = 0x7fffffff; s_lastkept = -1; }
        __syncthreads();
        float wbase = 0.f, total = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            if (w < warp) wbase += s_f[w];
            total += s_f[w];
        }
        uint32_t c[4] = {(uint32_t)slot, (uint32_t)a.draw_ctr[slot], 0u, 0u};
        philox4x32_10(c, ctl.seed_lo, ctl.seed_hi);
        const float target = (float)(c[0] >> 8) * (1.0f / 16777216.0f) * total;
        float cum = wbase + inc - loc;
        int mine = 0x7fffffff, lastk = -1;
        for (int k = k0; k < k1; ++k) {
            const float sc = lg[k] / T;
            if (top_k == 0 || order_key(sc) >= thr) {
                cum += expf(sc - smax);
                lastk = k;
                if (cum > target && mine == 0x7fffffff) mine = k;
            }
        }
        if (mine != 0x7fffffff) atomicMin(&s_pick, mine);
        if (lastk >= 0) atomicMax(&s_lastkept, lastk);
        __syncthreads();
        choice = s_pick != 0x7fffffff ? s_pick : (s_lastkept >= 0 ? s_lastkept : bi);
    }
    if (tid == 0) {
        a.tokens_out[r] = choice;
        if (pen) {
            float* cnt = a.rep_counts + (size_t)slot * V;
            int W = ctl.rep_window > REP_HIST_MAX ? REP_HIST_MAX : ctl.rep_window;
            if (W > 0) {
                int head = a.rep_head[slot], filled = a.rep_filled[slot];
                if (head >= W) head = 0;
                if (filled >= W) {
                    cnt[a.rep_hist[slot * REP_HIST_MAX + head]] -= 1.f;
                    filled = W;
                } else {
                    filled += 1;
                }
                a.rep_hist[slot * REP_HIST_MAX + head] = choice;
                a.rep_head[slot] = (head + 1) % W;
                a.rep_filled[slot] = filled;
            }
            cnt[choice] += 1.f;
        }
        a.draw_ctr[slot] += 1;
    }
}

}  // namespace vuib
