// Gated delta rule: a recurrent layer whose state per head is a matrix S (dim x vdim) in 32 bits,
//   S <- g S + k u^T,  u = beta (v - g S^T k),  o = S^T q            (S after the write)
// with unit queries and keys, a decay g and a step size beta per head and token.  Queries, keys and values pass a short
// causal convolution over time and silu first; the output is normed per head and gated.
//
// Both products with the state are taken before the write: with a = S^T k, b = S^T q and c = k . q of the old state,
//   u = beta (v - g a),  o = g b + c u,
// so a token needs one pass over S and one reduction.
//
// What a slot holds per layer, all fp32: S transposed (heads, vdp, dimp), a column of S contiguous; then a ring of the last
// `taps` rows of convolution inputs (taps, channels), the row of position p at p % taps.  One row more than the convolution
// looks back, so that a token's own row can be written while others read the rows before it.  A sequence that starts at
// position 0 starts from zeros, whatever the slot held before.
//
//   decode          k_delta_step: convolution, unit norms, gates, state, output norm and gate of one head and row.
//   many rows       k_delta_rows (convolution, unit norms, gates), the recurrence, then k_delta_gate (output norm and gate, the
//                   ring's new rows).  The recurrence runs token by token (k_delta_scan) or in chunks.
//
// Chunks of 64 tokens (bf16 models).  With G_t the sum of the log decays from the chunk's start to t and S_0 the state before
// it, unrolling the recurrence gives a unit lower triangular system for the chunk's writes,
//   (1 + A) u = beta v - (beta e^G k) S_0,   A_ts = beta_t e^(G_t - G_s) k_t . k_s  (s < t),
//   o_t = e^(G_t) S_0^T q_t + sum_{s <= t} e^(G_t - G_s) (k_s . q_t) u_s,   S_0' = e^(G_C) S_0 + sum_s e^(G_C - G_s) k_s u_s^T.
// k_delta_solve does what does not need S_0, every chunk on its own: it inverts 1 + A in fp32, gives U (right side beta v) and W
// (right side beta e^G k), and leaves P_ts = e^(G_t - G_s) q_t . k_s.  k_delta_chunks then carries the state
// from chunk to chunk: u = U - W S_0, o and S_0' as above.  The state stays in fp32 accumulators; a bf16 MMA takes a 32-bit
// operand as hi + lo bf16 pairs, three products per pair of operands (the product of the two low parts is left out).
#pragma once
#include "latent_attn.cuh"

namespace vuib {

constexpr int DR_MAX_DIM = 256;     // padded key size of a head
constexpr int DR_MAX_VDIM = 512;    // padded value size

struct DeltaShape {
    int H, G, dim, dimp, vdim, vdp, taps;
    int C;                 // convolution channels: G * dimp queries | G * dimp keys | H * vdp values
    int n_ab;              // first of H step-size columns and, after them, H decay columns of raw
    float scale, unit_eps, eps;
};

struct DeltaWeights {
    const float* conv;     // (taps, C), the last row multiplies the current token
    const float* neg_a;    // (H): -exp(A_log)
    const float* dt_bias;  // (H)
    const float* norm;     // (vdp)
};

struct DeltaState {
    float* base;           // slots
    size_t slot_floats, ring_off;
    __device__ __forceinline__ float* s(int slot, int h, const DeltaShape& d) const {
        return base + (size_t)slot * slot_floats + (size_t)h * d.vdp * d.dimp;
    }
    __device__ __forceinline__ float* ring(int slot) const { return base + (size_t)slot * slot_floats + ring_off; }
};

__device__ __forceinline__ float softplus32(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// (logarithm of the decay, step size) from a row of raw
__device__ __forceinline__ float2 delta_gates(const DeltaShape& d, const DeltaWeights& w, const float* raw, int h) {
    const float b = __ldcg(raw + d.n_ab + h), a = __ldcg(raw + d.n_ab + d.H + h);
    return make_float2(__ldg(w.neg_a + h) * softplus32(a + __ldg(w.dt_bias + h)), sigmoid32(b));
}

// Convolution and silu of channel c at position pos; the `back` rows before this one are raw rows of the same call.
__device__ __forceinline__ float delta_conv(const DeltaShape& d, const DeltaWeights& w, const float* raw, int ldraw, const float* ring,
                                            int pos, int back, int c) {
    float y = 0.f;
    for (int j0 = d.taps - 1; j0 >= 0; j0 -= 4) {
        float x[4], k[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int j = j0 - u;       // tokens back
            const bool in = j >= 0 && j <= pos;
            k[u] = in ? __ldg(w.conv + (size_t)(d.taps - 1 - j) * d.C + c) : 0.f;
            x[u] = !in ? 0.f : j <= back ? __ldcg(raw - (ptrdiff_t)j * ldraw + c) : __ldcg(ring + (size_t)((pos - j) % d.taps) * d.C + c);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) y = fmaf(x[u], k[u], y);
    }
    return silu32(y);
}

// ---------------------------------------------------------------------------
// Many rows, before the recurrence: out (M, C) unit queries (scaled) | unit keys | values; gates (M, H).
// ---------------------------------------------------------------------------
struct DeltaRowsArgs {
    DeltaShape d;
    DeltaWeights w;
    DeltaState st;
    const float* raw; int ldraw;
    float* out;
    float2* gates;
    const int32_t* row_slot;
    const int32_t* row_pos;
    const int2* row_ext;
};

// One row per CTA, any size.  SPLIT: queries and keys are left as bf16, a head's dimp high parts and then its dimp low parts,
// in the space of its floats.
template <bool SPLIT>
static __global__ void __launch_bounds__(LM_THREADS) k_delta_rows(DeltaRowsArgs a) {
    pdl_trigger();
    pdl_wait();
    const DeltaShape& d = a.d;
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slot = __ldcg(a.row_slot + m), pos = __ldcg(a.row_pos + m), back = __ldcg(&a.row_ext[m].x);
    const float* raw = a.raw + (size_t)m * a.ldraw;
    const float* ring = a.st.ring(slot);
    float* out = a.out + (size_t)m * d.C;
    constexpr int P = DR_MAX_DIM / 32;
    for (int i = warp; i < 2 * d.G; i += LM_WARPS) {
        float v[P], ss = 0.f;
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const int c = lane + 32 * j;
            v[j] = c < d.dimp ? delta_conv(d, a.w, raw, a.ldraw, ring, pos, back, i * d.dimp + c) : 0.f;
            ss = fmaf(v[j], v[j], ss);
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) + d.unit_eps) * (i < d.G ? d.scale : 1.0f);
#pragma unroll
        for (int j = 0; j < P; ++j)
            if (lane + 32 * j < d.dimp) {
                const int c = lane + 32 * j;
                if (SPLIT) {
                    bf16* o = reinterpret_cast<bf16*>(out + i * d.dimp);
                    const bf16 hi = f2bf(v[j] * r);
                    o[c] = hi;
                    o[d.dimp + c] = f2bf(v[j] * r - bf2f(hi));
                } else {
                    out[i * d.dimp + c] = v[j] * r;
                }
            }
    }
    for (int c = 2 * d.G * d.dimp + threadIdx.x; c < d.C; c += LM_THREADS) out[c] = delta_conv(d, a.w, raw, a.ldraw, ring, pos, back, c);
    for (int h = threadIdx.x; h < d.H; h += LM_THREADS) a.gates[(size_t)m * d.H + h] = delta_gates(d, a.w, raw, h);
}

// DR_ROWS consecutive rows and LM_WARPS heads per CTA, for up to DR_TAPS taps and heads of up to 128: the rows a convolution shares are read once.
constexpr int DR_ROWS = 8, DR_TAPS = 4;

template <bool SPLIT>
static __global__ void __launch_bounds__(LM_THREADS) k_delta_rows_tile(DeltaRowsArgs a, int M) {
    __shared__ int row_s[DR_ROWS], pos_s[DR_ROWS], back_s[DR_ROWS];
    pdl_trigger();
    const DeltaShape& d = a.d;
    const int m0 = blockIdx.x * DR_ROWS, nr = min(DR_ROWS, M - m0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_wait();
    if (threadIdx.x < DR_ROWS) {
        const int m = m0 + min((int)threadIdx.x, nr - 1);
        row_s[threadIdx.x] = __ldcg(a.row_slot + m);
        pos_s[threadIdx.x] = __ldcg(a.row_pos + m);
        back_s[threadIdx.x] = __ldcg(&a.row_ext[m].x);
    }
    __syncthreads();
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const int vblocks = (d.H * d.vdp + 127) / 128;
    const int i = blockIdx.y * LM_WARPS + warp;
    if (i < 2 * d.G + vblocks) {
        const bool unit = i < 2 * d.G;      // a query or key head; else 128 value columns
        const int c = unit ? i * d.dimp + 4 * lane : 2 * d.G * d.dimp + (i - 2 * d.G) * 128 + 4 * lane;
        const bool in = unit ? 4 * lane < d.dimp : c < d.C;
        float4 x[DR_ROWS + DR_TAPS - 1], w[DR_TAPS];
#pragma unroll
        for (int r = 0; r < DR_ROWS + DR_TAPS - 1; ++r) {
            const int m = m0 + r - (DR_TAPS - 1);
            x[r] = in && m >= 0 && m < M ? __ldcg(reinterpret_cast<const float4*>(a.raw + (size_t)m * a.ldraw + c)) : zero;
        }
#pragma unroll
        for (int j = 0; j < DR_TAPS; ++j)   // w[j] multiplies the row j back
            w[j] = in && j < d.taps ? __ldg(reinterpret_cast<const float4*>(a.w.conv + (size_t)(d.taps - 1 - j) * d.C + c)) : zero;
#pragma unroll
        for (int r = 0; r < DR_ROWS; ++r) {
            if (r >= nr) break;
            const int back = back_s[r], pos = pos_s[r];
            float4 y = zero;
#pragma unroll
            for (int j = DR_TAPS - 1; j >= 0; --j) {
                float4 v = x[r + DR_TAPS - 1 - j];
                if (j > back)                // before the portion: the ring, or nothing before the start
                    v = in && j < d.taps && j <= pos
                            ? __ldcg(reinterpret_cast<const float4*>(a.st.ring(row_s[r]) + (size_t)((pos - j) % d.taps) * d.C + c)) : zero;
                y.x = fmaf(v.x, w[j].x, y.x);
                y.y = fmaf(v.y, w[j].y, y.y);
                y.z = fmaf(v.z, w[j].z, y.z);
                y.w = fmaf(v.w, w[j].w, y.w);
            }
            y = make_float4(silu32(y.x), silu32(y.y), silu32(y.z), silu32(y.w));
            float* out = a.out + (size_t)(m0 + r) * d.C + (unit ? i * d.dimp : c);
            if (unit) {
                const float ss = warp_sum(fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, y.w * y.w))));
                const float n = 1.0f / sqrtf(ss + d.unit_eps) * (i < d.G ? d.scale : 1.0f);
                y = make_float4(y.x * n, y.y * n, y.z * n, y.w * n);
                if (SPLIT && in) {
                    uint2 hi, lo;
                    split_bf16x2(y.x, y.y, hi.x, lo.x);
                    split_bf16x2(y.z, y.w, hi.y, lo.y);
                    reinterpret_cast<uint2*>(out)[lane] = hi;
                    reinterpret_cast<uint2*>(out + d.dimp / 2)[lane] = lo;
                } else if (in) {
                    reinterpret_cast<float4*>(out)[lane] = y;
                }
            } else if (in) {
                *reinterpret_cast<float4*>(out) = y;
            }
        }
    }
    for (int i = blockIdx.y ? nr * d.H : (int)threadIdx.x; i < nr * d.H; i += LM_THREADS) {
        const int r = i / d.H, h = i - r * d.H;
        a.gates[(size_t)(m0 + r) * d.H + h] = delta_gates(d, a.w, a.raw + (size_t)(m0 + r) * a.ldraw, h);
    }
}

// ---------------------------------------------------------------------------
// The recurrence token by token.  LPC lanes share a column of S (NV float4 each); a lane group takes CP columns; nothing
// is exchanged between lane groups.  Grid: (portions, heads, blocks of columns).
// ---------------------------------------------------------------------------
constexpr int DS_THREADS = 128;
constexpr int DS_CP = 4;

struct DeltaScanArgs {
    DeltaShape d;
    DeltaState st;
    const float* x;           // k_delta_rows: out
    const float2* gates;
    const int4* segs;         // (slot, first position, rows, first row)
    float* o;                 // (M, H, vdp)
};

template <int LPC>
__device__ __forceinline__ float group_sum(float v) {
#pragma unroll
    for (int s = LPC / 2; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
    return v;
}
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
    return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc))));
}

template <int LPC, int NV>
static __global__ void __launch_bounds__(DS_THREADS) k_delta_scan(DeltaScanArgs a) {
    pdl_trigger();
    pdl_wait();
    const DeltaShape& d = a.d;
    constexpr int GROUPS = DS_THREADS / LPC;
    const int4 seg = a.segs[blockIdx.x];
    const int h = blockIdx.y, kvh = h / (d.H / d.G), sub = threadIdx.x % LPC, grp = threadIdx.x / LPC;
    const int c0 = (blockIdx.z * GROUPS + grp) * DS_CP;
    const bool live = c0 < d.vdp;          // vdp is a multiple of DS_CP
    float* S = a.st.s(seg.x, h, d) + (size_t)(live ? c0 : 0) * d.dimp;
    const int nv = d.dimp / 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 s[DS_CP][NV];
#pragma unroll
    for (int c = 0; c < DS_CP; ++c)
#pragma unroll
        for (int i = 0; i < NV; ++i)
            s[c][i] = seg.y > 0 && sub + i * LPC < nv ? __ldcg(reinterpret_cast<const float4*>(S + (size_t)c * d.dimp) + sub + i * LPC) : zero;
    float4 k[NV], q[NV], v;
    float2 gt;
    auto load = [&](int m) {
        const float* x = a.x + (size_t)m * d.C;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const bool in = sub + i * LPC < nv;
            q[i] = in ? __ldcg(reinterpret_cast<const float4*>(x + kvh * d.dimp) + sub + i * LPC) : zero;
            k[i] = in ? __ldcg(reinterpret_cast<const float4*>(x + (d.G + kvh) * d.dimp) + sub + i * LPC) : zero;
        }
        v = __ldcg(reinterpret_cast<const float4*>(x + 2 * d.G * d.dimp + h * d.vdp + (live ? c0 : 0)));
        gt = __ldcg(a.gates + (size_t)m * d.H + h);
    };
    load(seg.w);
    for (int n = 0; n < seg.z; ++n) {
        float4 kc[NV], qc[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) { kc[i] = k[i]; qc[i] = q[i]; }
        const float vv[DS_CP] = {v.x, v.y, v.z, v.w};
        const float g = expf(gt.x), beta = gt.y;
        if (n + 1 < seg.z) load(seg.w + n + 1);
        float r[2 * DS_CP + 1] = {};
#pragma unroll
        for (int i = 0; i < NV; ++i) {
#pragma unroll
            for (int c = 0; c < DS_CP; ++c) {
                r[c] = dot4(s[c][i], kc[i], r[c]);
                r[DS_CP + c] = dot4(s[c][i], qc[i], r[DS_CP + c]);
            }
            r[2 * DS_CP] = dot4(kc[i], qc[i], r[2 * DS_CP]);
        }
#pragma unroll
        for (int j = 0; j < 2 * DS_CP + 1; ++j) r[j] = group_sum<LPC>(r[j]);
        float o[DS_CP];
#pragma unroll
        for (int c = 0; c < DS_CP; ++c) {
            const float u = beta * (vv[c] - g * r[c]);
            o[c] = fmaf(g, r[DS_CP + c], r[2 * DS_CP] * u);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                s[c][i].x = fmaf(g, s[c][i].x, kc[i].x * u);
                s[c][i].y = fmaf(g, s[c][i].y, kc[i].y * u);
                s[c][i].z = fmaf(g, s[c][i].z, kc[i].z * u);
                s[c][i].w = fmaf(g, s[c][i].w, kc[i].w * u);
            }
        }
        if (live && sub == 0)
            *reinterpret_cast<float4*>(a.o + ((size_t)(seg.w + n) * d.H + h) * d.vdp + c0) = make_float4(o[0], o[1], o[2], o[3]);
    }
    if (live)
#pragma unroll
        for (int c = 0; c < DS_CP; ++c)
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (sub + i * LPC < nv) *(reinterpret_cast<float4*>(S + (size_t)c * d.dimp) + sub + i * LPC) = s[c][i];
}

// ---------------------------------------------------------------------------
// The chunked form.
// ---------------------------------------------------------------------------
constexpr int DC_ROWS = 64;
constexpr int DC_MAX_DIM = 128;   // padded key size
constexpr int DC_LDP = DC_ROWS + 8;
constexpr int DC_LDA = DC_ROWS + 4;

struct DeltaChunkArgs {
    DeltaShape d;
    DeltaState st;
    const float* x;           // k_delta_rows<true>: out
    const float2* gates;
    const int4* tiles;        // 2 per chunk; the first: (first row, rows, slot, first position)
    const int4* segs;         // (slot, first position, rows, first row)
    bf16* w;                  // (M, H, 2, dimp): high and low parts of W
    float* u;                 // (M, H, vdp)
    bf16* p;                  // (M, H, 2, 64)
    float* o;                 // (M, H, vdp)
    FastDiv row_vecs;         // dimp / 4: 16-byte pieces of a row's high and low parts
};

// 64 rows of [high | low] parts, n of them valid, into two tiles of padded rows.
__device__ __forceinline__ void dc_fetch(bf16* dst, const bf16* src, size_t stride, int n, int dimp, const FastDiv& vecs, int n_vecs) {
    const int ld = dimp + 8, half = n_vecs / 2;
    for (int i = threadIdx.x; i < DC_ROWS * n_vecs; i += LM_THREADS) {
        const int r = vecs.div(i), v = i - r * n_vecs;
        bf16* to = dst + (v < half ? r * ld + v * 8 : (DC_ROWS + r) * ld + (v - half) * 8);
        cp_async16(to, src + (r < n ? (size_t)r * stride + v * 8 : 0), r < n);
    }
}

// d += a b with a and b as (high, low) pairs
__device__ __forceinline__ void mma_split(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1,
                                          uint32_t bl0, uint32_t bl1) {
    mma_bf16(d, ah, bh0, bh1);
    mma_bf16(d, ah, bl0, bl1);
    mma_bf16(d, al, bh0, bh1);
}

constexpr int DC_VCOLS = 128;     // value columns of k_delta_solve in shared memory at a time
constexpr int DC_LDB = DC_VCOLS + 8;
constexpr size_t DC_T_BYTES = (size_t)2 * DC_ROWS * DC_LDP * 2;   // a 64 x 64 matrix as (high, low) parts; more than one of floats
static inline size_t delta_solve_smem(int dimp) {
    return (size_t)2 * DC_ROWS * (dimp + 8) * 2 + (size_t)2 * DC_ROWS * DC_LDB * 2 + 2 * DC_T_BYTES;
}

// CTA = (chunk, head).  T = (1 + A)^-1 by blocks of 16: the diagonal ones by substitution, a thread per column; the others from
//   T_ij = -T_ii sum_{j <= k < i} A_ik T_kj
// one subdiagonal after the other.  Then W = T (beta e^G k) and U = T (beta v) on the tensor cores, the factors of a token moved into
// T's column.
static __global__ void __launch_bounds__(LM_THREADS, 2) k_delta_solve(DeltaChunkArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float G[DC_ROWS], beta[DC_ROWS];
    pdl_trigger();
    const DeltaShape& d = a.d;
    const int ld = d.dimp + 8, nvec = d.dimp / 4;
    bf16* Ks = reinterpret_cast<bf16*>(smem_raw);              // [2][64][ld]
    bf16* Bs = Ks + (size_t)2 * DC_ROWS * ld;                  // queries [2][64][ld], then values [2][64][DC_LDB]
    unsigned char* t0 = reinterpret_cast<unsigned char*>(Bs + (size_t)2 * DC_ROWS * DC_LDB);
    float* A = reinterpret_cast<float*>(t0);                   // [t][s], s < t
    float* T = reinterpret_cast<float*>(t0 + DC_T_BYTES);      // [t][s], s <= t by blocks; blocks above hold what is on its way
    bf16* Tw = reinterpret_cast<bf16*>(t0);                    // T with columns times beta e^G, [2][64][DC_LDP]
    bf16* Tu = reinterpret_cast<bf16*>(t0 + DC_T_BYTES);       // T with columns times beta
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, kvh = h / (d.H / d.G);
    pdl_wait();
    const int4 tile = a.tiles[2 * blockIdx.x];
    const int row0 = tile.x, n = tile.y;
    const float* x = a.x + (size_t)row0 * d.C;
    dc_fetch(Ks, reinterpret_cast<const bf16*>(x + (d.G + kvh) * d.dimp), 2 * d.C, n, d.dimp, a.row_vecs, nvec);
    dc_fetch(Bs, reinterpret_cast<const bf16*>(x + kvh * d.dimp), 2 * d.C, n, d.dimp, a.row_vecs, nvec);
    cp_async_commit();
    if (warp == 0) {
        float2 gt[2];
#pragma unroll
        for (int i = 0; i < 2; ++i)
            gt[i] = 2 * lane + i < n ? __ldcg(a.gates + (size_t)(row0 + 2 * lane + i) * d.H + h) : make_float2(0.f, 0.f);
        float sum = gt[0].x + gt[1].x;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += v;
        }
        G[2 * lane] = sum - gt[1].x;
        G[2 * lane + 1] = sum;
        beta[2 * lane] = gt[0].y;
        beta[2 * lane + 1] = gt[1].y;
    }
    cp_async_wait<0>();
    __syncthreads();
    {   // warps 0-3: keys with keys, 4-7: queries with keys; 16 rows each, columns up to the diagonal
        const int mt = warp & 3;
        const bool is_q = warp >= 4;
        const bf16* P = (is_q ? Bs : Ks) + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + (lane >> 4) * 8;
        const bf16* K = Ks + ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8;
        float acc[4][2][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[j][0][i] = acc[j][1][i] = 0.f;
        for (int ks = 0; ks < d.dimp / 16; ++ks) {
            uint32_t ah[4], al[4];
            ldsm_x4(ah, P + ks * 16);
            ldsm_x4(al, P + DC_ROWS * ld + ks * 16);
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (j <= mt) {
                    uint32_t bh[4], bl[4];
                    ldsm_x4(bh, K + j * 16 * ld + ks * 16);
                    ldsm_x4(bl, K + (DC_ROWS + j * 16) * ld + ks * 16);
                    mma_split(acc[j][0], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma_split(acc[j][1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (j <= mt)
#pragma unroll
                for (int half = 0; half < 2; ++half)
#pragma unroll
                    for (int hi = 0; hi < 2; ++hi) {
                        const int r = mt * 16 + g + hi * 8, c = j * 16 + half * 8 + 2 * t;
                        const float v0 = c <= r ? expf(G[r] - G[c]) * acc[j][half][2 * hi] : 0.f;
                        const float v1 = c + 1 <= r ? expf(G[r] - G[c + 1]) * acc[j][half][2 * hi + 1] : 0.f;
                        if (!is_q) {
                            *reinterpret_cast<float2*>(A + r * DC_LDA + c) = make_float2(c < r ? beta[r] * v0 : 0.f, c + 1 < r ? beta[r] * v1 : 0.f);
                        } else if (r < n) {
                            uint32_t ph, pl;
                            split_bf16x2(v0, v1, ph, pl);
                            bf16* p = a.p + ((size_t)(row0 + r) * d.H + h) * 2 * DC_ROWS + c;
                            *reinterpret_cast<uint32_t*>(p) = ph;
                            *reinterpret_cast<uint32_t*>(p + DC_ROWS) = pl;
                        }
                    }
    }
    __syncthreads();
    // the values of columns v0 .. v0 + 127, by threads first, first + step, ...
    auto values = [&](int v0, int first, int step) {
        const float* v = x + 2 * d.G * d.dimp + h * d.vdp + v0;
        const int cols = min(DC_VCOLS, d.vdp - v0);
        constexpr int U = 4;
        for (int i0 = first; i0 < DC_ROWS * (DC_VCOLS / 4); i0 += U * step) {
            float4 f[U];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * step, r = i / (DC_VCOLS / 4), c = i % (DC_VCOLS / 4) * 4;
                f[u] = r < n && c < cols ? __ldcg(reinterpret_cast<const float4*>(v + (size_t)r * d.C + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * step, r = i / (DC_VCOLS / 4), c = i % (DC_VCOLS / 4) * 4;
                if (r < DC_ROWS) {
                    uint2 hi, lo;
                    split_bf16x2(f[u].x, f[u].y, hi.x, lo.x);
                    split_bf16x2(f[u].z, f[u].w, hi.y, lo.y);
                    *reinterpret_cast<uint2*>(Bs + r * DC_LDB + c) = hi;
                    *reinterpret_cast<uint2*>(Bs + (DC_ROWS + r) * DC_LDB + c) = lo;
                }
            }
        }
    };
    if (warp < 2) {
        const int b = tid & ~15, c = tid & 15;     // block at row b, column c of it
        float v[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            v[i] = i == c ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) v[i] = fmaf(-A[(b + i) * DC_LDA + b + j], v[j], v[i]);
            T[(b + i) * DC_LDA + b + c] = v[i];
        }
    } else {
        values(0, tid - 64, LM_THREADS - 64);
    }
    __syncthreads();
    {
        const int r = tid >> 4, c = tid & 15;
        for (int diag = 1; diag < 4; ++diag) {
            for (int j = 0; j + diag < 4; ++j) {   // sum_k A_ik T_kj, left in the block above the diagonal
                const int i = j + diag;
                float v = 0.f;
                for (int k = 16 * j; k < 16 * i; ++k) v = fmaf(A[(16 * i + r) * DC_LDA + k], T[k * DC_LDA + 16 * j + c], v);
                T[(16 * j + r) * DC_LDA + 16 * i + c] = v;
            }
            __syncthreads();
            for (int j = 0; j + diag < 4; ++j) {
                const int i = j + diag;
                float v = 0.f;
#pragma unroll
                for (int k = 0; k < 16; ++k) v = fmaf(T[(16 * i + r) * DC_LDA + 16 * i + k], T[(16 * j + k) * DC_LDA + 16 * i + c], v);
                T[(16 * i + r) * DC_LDA + 16 * j + c] = -v;
            }
            __syncthreads();
        }
    }
    {   // T, scaled, to its (high, low) parts; a thread takes 16 columns of a row
        const int r = tid >> 2, c0 = (tid & 3) * 16;
        __align__(16) float v[16];
#pragma unroll
        for (int i = 0; i < 16; i += 4) *reinterpret_cast<float4*>(v + i) = *reinterpret_cast<const float4*>(T + r * DC_LDA + c0 + i);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
            const int c = c0 + i;
            const float b0 = v[i] * beta[c], b1 = v[i + 1] * beta[c + 1];
            uint32_t hi, lo;
            split_bf16x2(b0, b1, hi, lo);
            *reinterpret_cast<uint32_t*>(Tu + r * DC_LDP + c) = hi;
            *reinterpret_cast<uint32_t*>(Tu + (DC_ROWS + r) * DC_LDP + c) = lo;
            split_bf16x2(b0 * expf(G[c]), b1 * expf(G[c + 1]), hi, lo);
            *reinterpret_cast<uint32_t*>(Tw + r * DC_LDP + c) = hi;
            *reinterpret_cast<uint32_t*>(Tw + (DC_ROWS + r) * DC_LDP + c) = lo;
        }
        __syncthreads();
    }
    // a warp takes 16 columns of W or U at a time
    const int a_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * DC_LDP + (lane >> 4) * 8;
    auto product = [&](const bf16* M, const bf16* B, int ldb, auto put) {
        uint32_t bh[4][4], bl[4][4];
        const bf16* b = B + ((lane & 7) + ((lane >> 3) & 1) * 8) * ldb + (lane >> 4) * 8;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            ldsm_x4_t(bh[ks], b + ks * 16 * ldb);
            ldsm_x4_t(bl[ks], b + (DC_ROWS + ks * 16) * ldb);
        }
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
            float acc[2][4] = {};
#pragma unroll
            for (int ks = 0; ks <= mt; ++ks) {
                uint32_t ah[4], al[4];
                ldsm_x4(ah, M + a_off + mt * 16 * DC_LDP + ks * 16);
                ldsm_x4(al, M + a_off + (DC_ROWS + mt * 16) * DC_LDP + ks * 16);
                mma_split(acc[0], ah, al, bh[ks][0], bh[ks][1], bl[ks][0], bl[ks][1]);
                mma_split(acc[1], ah, al, bh[ks][2], bh[ks][3], bl[ks][2], bl[ks][3]);
            }
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    const int r = mt * 16 + g + hi * 8;
                    if (r < n) put((size_t)(row0 + r) * d.H + h, half * 8 + 2 * t, acc[half][2 * hi], acc[half][2 * hi + 1]);
                }
        }
    };
    const int w_items = d.dimp / 16;
    for (int v0 = 0; v0 < d.vdp; v0 += DC_VCOLS) {
        if (v0) {
            __syncthreads();
            values(v0, tid, LM_THREADS);
            __syncthreads();
        }
        const int first = v0 ? w_items : 0, items = w_items + min(DC_VCOLS, d.vdp - v0) / 16;
        for (int it = first + warp; it < items; it += LM_WARPS) {
            if (it < w_items) {
                product(Tw, Ks + it * 16, ld, [&](size_t row, int c, float p0, float p1) {
                    uint32_t hi, lo;
                    split_bf16x2(p0, p1, hi, lo);
                    bf16* w = a.w + row * 2 * d.dimp + it * 16 + c;
                    *reinterpret_cast<uint32_t*>(w) = hi;
                    *reinterpret_cast<uint32_t*>(w + d.dimp) = lo;
                });
            } else {
                product(Tu, Bs + (it - w_items) * 16, DC_LDB, [&](size_t row, int c, float p0, float p1) {
                    *reinterpret_cast<float2*>(a.u + row * d.vdp + v0 + (it - w_items) * 16 + c) = make_float2(p0, p1);
                });
            }
        }
    }
}

template <int NB>
static inline size_t delta_chunks_smem(int dimp) {
    return ((size_t)3 * 2 * DC_ROWS * (dimp + 8) + (size_t)2 * DC_ROWS * DC_LDP + (size_t)2 * NB * (dimp + 8) + (size_t)4 * DC_ROWS * (NB + 8)) * 2 +
           (size_t)DC_ROWS * (NB + 4) * 4;
}

// CTA = (portion, head, NB value columns).  A warp keeps 16 rows of the state as MMA accumulators.  W, q, U of the next chunk
// are fetched while this chunk's second half runs, k and P while the next chunk's first half does.
template <int NB>
static __global__ void __launch_bounds__(LM_THREADS) k_delta_chunks(DeltaChunkArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float eg[DC_ROWS], eg_rest[DC_ROWS];   // e^G_t, e^(G_C - G_t)
    constexpr int NT = NB / 8, LDV = NB + 8, LDU = NB + 4;
    pdl_trigger();
    const DeltaShape& d = a.d;
    const int ld = d.dimp + 8, nvec = d.dimp / 4, ks_dim = d.dimp / 16;
    bf16* Ws = reinterpret_cast<bf16*>(smem_raw);      // [2][64][ld], high and low
    bf16* Qs = Ws + (size_t)2 * DC_ROWS * ld;
    bf16* Ks = Qs + (size_t)2 * DC_ROWS * ld;
    bf16* Ps = Ks + (size_t)2 * DC_ROWS * ld;          // [2][64][DC_LDP]
    bf16* Ss = Ps + (size_t)2 * DC_ROWS * DC_LDP;      // [2][NB][ld], the state by columns
    bf16* Vs = Ss + (size_t)2 * NB * ld;               // [2][64][LDV]: u
    bf16* Vd = Vs + (size_t)2 * DC_ROWS * LDV;         // the same times e^(G_C - G_t)
    float* Us = reinterpret_cast<float*>(Vd + (size_t)2 * DC_ROWS * LDV);   // [64][LDU]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, kvh = h / (d.H / d.G), c0 = blockIdx.z * NB, nc = min(NB, d.vdp - c0);   // nc is a multiple of 16
    pdl_wait();
    const int4 seg = a.segs[blockIdx.x];
    const int n_chunks = (seg.z + DC_ROWS - 1) / DC_ROWS;
    auto fetch_first = [&](int ci) {       // W, q, U
        if (ci < n_chunks) {
            const int row0 = seg.w + ci * DC_ROWS, n = min(DC_ROWS, seg.z - ci * DC_ROWS);
            dc_fetch(Ws, a.w + ((size_t)row0 * d.H + h) * 2 * d.dimp, (size_t)2 * d.H * d.dimp, n, d.dimp, a.row_vecs, nvec);
            dc_fetch(Qs, reinterpret_cast<const bf16*>(a.x + (size_t)row0 * d.C + kvh * d.dimp), 2 * d.C, n, d.dimp, a.row_vecs, nvec);
            for (int i = tid; i < DC_ROWS * (NB / 4); i += LM_THREADS) {
                const int r = i / (NB / 4), v = i % (NB / 4);
                const bool ok = r < n && 4 * v < nc;
                cp_async16(Us + r * LDU + v * 4, a.u + (ok ? ((size_t)(row0 + r) * d.H + h) * d.vdp + c0 + v * 4 : 0), ok);
            }
        }
        cp_async_commit();
    };
    auto fetch_second = [&](int ci) {      // k, P
        if (ci < n_chunks) {
            const int row0 = seg.w + ci * DC_ROWS, n = min(DC_ROWS, seg.z - ci * DC_ROWS);
            dc_fetch(Ks, reinterpret_cast<const bf16*>(a.x + (size_t)row0 * d.C + (d.G + kvh) * d.dimp), 2 * d.C, n, d.dimp, a.row_vecs, nvec);
            for (int i = tid; i < DC_ROWS * 16; i += LM_THREADS) {
                const int r = i >> 4, v = i & 15;
                cp_async16(Ps + ((v >> 3) * DC_ROWS + r) * DC_LDP + (v & 7) * 8,
                           a.p + (r < n ? ((size_t)(row0 + r) * d.H + h) * 2 * DC_ROWS + v * 8 : 0), r < n);
            }
        }
        cp_async_commit();
    };
    float lg[2];                           // warp 0: log decays of rows 2 * lane, 2 * lane + 1
    auto ask_gates = [&](int ci) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = ci * DC_ROWS + 2 * lane + i;
            lg[i] = warp == 0 && r < seg.z ? __ldcg(a.gates + (size_t)(seg.w + r) * d.H + h).x : 0.f;
        }
    };
    fetch_first(0);
    fetch_second(0);
    ask_gates(0);
    // the state: rows warp * 16 + g (+ 8), columns c0 + nt * 8 + 2 * t (+ 1)
    const bool has_s = warp < ks_dim;
    float* S = a.st.s(seg.x, h, d) + (size_t)c0 * d.dimp + warp * 16 + g;
    float s[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int col = i * 8 + 2 * t + (e & 1);
            s[i][e] = has_s && seg.y > 0 && col < nc ? __ldcg(S + (size_t)col * d.dimp + (e >> 1) * 8) : 0.f;
        }
    const int mt = warp & 3;
    const int a_off = (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + (lane >> 4) * 8;
    const int b_off = ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8;
    const int v_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8;
    const int kt_off = ((lane & 7) + ((lane >> 4) & 1) * 8) * ld + warp * 16 + ((lane >> 3) & 1) * 8;
    for (int ci = 0; ci < n_chunks; ++ci) {
        const int row0 = seg.w + ci * DC_ROWS, n = min(DC_ROWS, seg.z - ci * DC_ROWS);
        if (has_s)
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    bf16* p = Ss + (i * 8 + 2 * t + (e & 1)) * ld + warp * 16 + g + (e >> 1) * 8;
                    const bf16 hi = f2bf(s[i][e]);
                    p[0] = hi;
                    p[NB * ld] = f2bf(s[i][e] - bf2f(hi));
                }
        if (warp == 0) {
            float sum = lg[0] + lg[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += v;
            }
            const float total = __shfl_sync(0xffffffffu, sum, 31), first = sum - lg[1];
            eg[2 * lane] = expf(first);
            eg[2 * lane + 1] = expf(sum);
            eg_rest[2 * lane] = expf(total - first);
            eg_rest[2 * lane + 1] = expf(total - sum);
        }
        ask_gates(ci + 1);
        cp_async_wait<1>();
        __syncthreads();
        // ---- W S (warps 0-3), q S (warps 4-7)
        float acc[NT][4];
#pragma unroll
        for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
        {
            const bf16* A = (warp < 4 ? Ws : Qs) + a_off;
#pragma unroll 2
            for (int ks = 0; ks < ks_dim; ++ks) {
                uint32_t ah[4], al[4];
                ldsm_x4(ah, A + ks * 16);
                ldsm_x4(al, A + DC_ROWS * ld + ks * 16);
#pragma unroll
                for (int j = 0; j < NT / 2; ++j) {
                    uint32_t bh[4], bl[4];
                    ldsm_x4(bh, Ss + b_off + j * 16 * ld + ks * 16);
                    ldsm_x4(bl, Ss + b_off + (NB + j * 16) * ld + ks * 16);
                    mma_split(acc[2 * j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma_split(acc[2 * j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
            }
        }
        const int r_lo = mt * 16 + g, r_hi = r_lo + 8;
        if (warp < 4) {
            const float d_lo = eg_rest[r_lo], d_hi = eg_rest[r_hi];
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    const int r = hi ? r_hi : r_lo, c = i * 8 + 2 * t;
                    const float dd = hi ? d_hi : d_lo;
                    const float2 u = *reinterpret_cast<const float2*>(Us + r * LDU + c);
                    const float u0 = u.x - acc[i][2 * hi], u1 = u.y - acc[i][2 * hi + 1];
                    uint32_t vh, vl;
                    split_bf16x2(u0, u1, vh, vl);
                    *reinterpret_cast<uint32_t*>(Vs + r * LDV + c) = vh;
                    *reinterpret_cast<uint32_t*>(Vs + (DC_ROWS + r) * LDV + c) = vl;
                    split_bf16x2(u0 * dd, u1 * dd, vh, vl);
                    *reinterpret_cast<uint32_t*>(Vd + r * LDV + c) = vh;
                    *reinterpret_cast<uint32_t*>(Vd + (DC_ROWS + r) * LDV + c) = vl;
                }
        } else {
            const float e_lo = eg[r_lo], e_hi = eg[r_hi];
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                acc[i][0] *= e_lo; acc[i][1] *= e_lo;
                acc[i][2] *= e_hi; acc[i][3] *= e_hi;
            }
        }
        cp_async_wait<0>();      // k and P
        const float decay = eg[DC_ROWS - 1];
        __syncthreads();
        fetch_first(ci + 1);
        // ---- S = e^G_C S + k^T u
        if (has_s) {
#pragma unroll
            for (int i = 0; i < NT; ++i) { s[i][0] *= decay; s[i][1] *= decay; s[i][2] *= decay; s[i][3] *= decay; }
#pragma unroll
            for (int ks = 0; ks < DC_ROWS / 16; ++ks) {
                uint32_t ah[4], al[4];
                ldsm_x4_t(ah, Ks + kt_off + ks * 16 * ld);
                ldsm_x4_t(al, Ks + kt_off + (DC_ROWS + ks * 16) * ld);
#pragma unroll
                for (int j = 0; j < NT / 2; ++j) {
                    uint32_t bh[4], bl[4];
                    ldsm_x4_t(bh, Vd + v_off + ks * 16 * LDV + j * 16);
                    ldsm_x4_t(bl, Vd + v_off + (DC_ROWS + ks * 16) * LDV + j * 16);
                    mma_split(s[2 * j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma_split(s[2 * j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
            }
        }
        // ---- o = e^G q S + P u
        if (warp >= 4) {
            const bf16* A = Ps + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * DC_LDP + (lane >> 4) * 8;
#pragma unroll
            for (int ks = 0; ks < DC_ROWS / 16; ++ks)
                if (ks <= mt) {
                    uint32_t ah[4], al[4];
                    ldsm_x4(ah, A + ks * 16);
                    ldsm_x4(al, A + DC_ROWS * DC_LDP + ks * 16);
#pragma unroll
                    for (int j = 0; j < NT / 2; ++j) {
                        uint32_t bh[4], bl[4];
                        ldsm_x4_t(bh, Vs + v_off + ks * 16 * LDV + j * 16);
                        ldsm_x4_t(bl, Vs + v_off + (DC_ROWS + ks * 16) * LDV + j * 16);
                        mma_split(acc[2 * j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                        mma_split(acc[2 * j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                    }
                }
#pragma unroll
            for (int i = 0; i < NT; ++i)
                if (i * 8 < nc) {
                    float* o = a.o + ((size_t)row0 * d.H + h) * d.vdp + c0 + i * 8 + 2 * t;
                    if (r_lo < n) *reinterpret_cast<float2*>(o + (size_t)r_lo * d.H * d.vdp) = make_float2(acc[i][0], acc[i][1]);
                    if (r_hi < n) *reinterpret_cast<float2*>(o + (size_t)r_hi * d.H * d.vdp) = make_float2(acc[i][2], acc[i][3]);
                }
        }
        __syncthreads();         // k, P, u and the state's tiles are used up
        fetch_second(ci + 1);
    }
    if (has_s)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int col = i * 8 + 2 * t + (e & 1);
                if (col < nc) S[(size_t)col * d.dimp + (e >> 1) * 8] = s[i][e];
            }
}

// ---------------------------------------------------------------------------
// Many rows, after the recurrence: output norm and gate per head, and the last rows of a portion into the ring.
// ---------------------------------------------------------------------------
template <class T>
struct DeltaGateArgs {
    DeltaShape d;
    DeltaWeights w;
    DeltaState st;
    const float* raw; int ldraw;
    const float* o;           // (M, H, vdp)
    const T* gate; int ldgate;
    T* out; int ldo;
    const int32_t* row_slot;
    const int32_t* row_pos;
    const int2* row_ext;
};

// A warp takes U (row, head) pairs at a time, P * 128 columns of each.
template <class T, int P, int U>
static __global__ void __launch_bounds__(LM_THREADS) k_delta_gate(DeltaGateArgs<T> a, int M) {
    pdl_trigger();
    const DeltaShape& d = a.d;
    const int lane = threadIdx.x & 31, i0 = (blockIdx.x * LM_WARPS + (threadIdx.x >> 5)) * U, n = M * d.H;
    float4 w[P];
#pragma unroll
    for (int j = 0; j < P; ++j) w[j] = 4 * lane + 128 * j < d.vdp ? __ldg(reinterpret_cast<const float4*>(a.w.norm) + lane + 32 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_wait();
    float4 v[U][P];
    float gt[U][P][4];
    int left[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int i = min(i0 + u, n - 1), m = i / d.H, h = i - m * d.H;
        left[u] = __ldcg(&a.row_ext[m].y);
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const int c = 4 * lane + 128 * j;
            const bool in = c < d.vdp;
            v[u][j] = in ? __ldcg(reinterpret_cast<const float4*>(a.o + (size_t)i * d.vdp + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
            Store<T>::ld4(a.gate + (size_t)m * a.ldgate + h * d.vdp + (in ? c : 0), gt[u][j]);
        }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
        if (i0 + u >= n) break;
        const int i = i0 + u, m = i / d.H, h = i - m * d.H;
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < P; ++j) ss = dot4(v[u][j], v[u][j], ss);
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)d.vdim + d.eps);
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const int c = 4 * lane + 128 * j;
            if (c < d.vdp)
                Store<T>::put4(a.out + (size_t)m * a.ldo + h * d.vdp + c,
                               make_float4(v[u][j].x * r * w[j].x * gt[u][j][0], v[u][j].y * r * w[j].y * gt[u][j][1],
                                           v[u][j].z * r * w[j].z * gt[u][j][2], v[u][j].w * r * w[j].w * gt[u][j][3]));
        }
        if (left[u] < d.taps) {           // this head's share of the row's channels
            const int share = (d.C / 4 + d.H - 1) / d.H, end = min(d.C / 4, (h + 1) * share);
            const float4* raw = reinterpret_cast<const float4*>(a.raw + (size_t)m * a.ldraw);
            float4* ring = reinterpret_cast<float4*>(a.st.ring(__ldcg(a.row_slot + m)) + (size_t)(__ldcg(a.row_pos + m) % d.taps) * d.C);
            for (int c0 = h * share + lane; c0 < end; c0 += 4 * 32) {
                float4 t[4];
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (c0 + 32 * j < end) t[j] = __ldcg(raw + c0 + 32 * j);
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (c0 + 32 * j < end) ring[c0 + 32 * j] = t[j];
            }
        }
    }
}

// ---------------------------------------------------------------------------
// One token of one row and head: everything between the two matrix products.  The CTA's lane groups take the columns in
// turn; the first CP columns of a group are requested before the convolution.
// ---------------------------------------------------------------------------
constexpr int DT_THREADS = 512;
constexpr int DT_CP = 8;

template <class T, int LPC, int NV>
static __global__ void __launch_bounds__(DT_THREADS) k_delta_step(DeltaGateArgs<T> a) {
    __shared__ __align__(16) float qk_s[2][DR_MAX_DIM];
    __shared__ float v_s[DR_MAX_VDIM], o_s[DR_MAX_VDIM];
    pdl_trigger();
    const DeltaShape& d = a.d;
    constexpr int GROUPS = DT_THREADS / LPC;
    const int h = blockIdx.x, m = blockIdx.y, rep = d.H / d.G, kvh = h / rep;
    const int tid = threadIdx.x, lane = tid & 31, sub = tid % LPC, grp = tid / LPC;
    const int nv = d.dimp / 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_wait();
    const int slot = __ldcg(a.row_slot + m), pos = __ldcg(a.row_pos + m);
    float* S = a.st.s(slot, h, d);
    float4 s[DT_CP][NV];
    auto load = [&](int b) {
#pragma unroll
        for (int c = 0; c < DT_CP; ++c) {
            const int col = (b * DT_CP + c) * GROUPS + grp;
#pragma unroll
            for (int i = 0; i < NV; ++i)
                s[c][i] = pos > 0 && col < d.vdp && sub + i * LPC < nv ? __ldcg(reinterpret_cast<const float4*>(S + (size_t)col * d.dimp) + sub + i * LPC) : zero;
        }
    };
    load(0);
    const float* raw = a.raw + (size_t)m * a.ldraw;
    const float2 gt = delta_gates(d, a.w, raw, h);
    {   // convolution of this head's channels; every channel's row goes into the ring once
        float* ring = a.st.ring(slot);
        float* own = ring + (size_t)(pos % d.taps) * d.C;
        for (int i = tid; i < 2 * d.dimp + d.vdp; i += DT_THREADS) {
            const int part = i < d.dimp ? 0 : i < 2 * d.dimp ? 1 : 2, e = i - part * d.dimp;
            const int c = part < 2 ? (part * d.G + kvh) * d.dimp + e : 2 * d.G * d.dimp + h * d.vdp + e;
            const float y = delta_conv(d, a.w, raw, 0, ring, pos, 0, c);
            if (part < 2) qk_s[part][e] = y;
            else v_s[e] = y;
            if (part == 2 || h % rep == 0) own[c] = __ldcg(raw + c);
        }
    }
    __syncthreads();
    float4 q[NV], k[NV];
    float qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const bool in = sub + i * LPC < nv;
        q[i] = in ? reinterpret_cast<const float4*>(qk_s[0])[sub + i * LPC] : zero;
        k[i] = in ? reinterpret_cast<const float4*>(qk_s[1])[sub + i * LPC] : zero;
        qq = dot4(q[i], q[i], qq);
        kk = dot4(k[i], k[i], kk);
        kq = dot4(k[i], q[i], kq);
    }
    const float rq = 1.0f / sqrtf(group_sum<LPC>(qq) + d.unit_eps) * d.scale, rk = 1.0f / sqrtf(group_sum<LPC>(kk) + d.unit_eps);
    kq = group_sum<LPC>(kq) * rq * rk;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        q[i].x *= rq; q[i].y *= rq; q[i].z *= rq; q[i].w *= rq;
        k[i].x *= rk; k[i].y *= rk; k[i].z *= rk; k[i].w *= rk;
    }
    const float g = expf(gt.x), beta = gt.y;
    for (int b = 0; b * DT_CP * GROUPS < d.vdp; ++b) {
        if (b) load(b);
        float r[2 * DT_CP] = {};
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int c = 0; c < DT_CP; ++c) {
                r[c] = dot4(s[c][i], k[i], r[c]);
                r[DT_CP + c] = dot4(s[c][i], q[i], r[DT_CP + c]);
            }
#pragma unroll
        for (int j = 0; j < 2 * DT_CP; ++j) r[j] = group_sum<LPC>(r[j]);
#pragma unroll
        for (int c = 0; c < DT_CP; ++c) {
            const int col = (b * DT_CP + c) * GROUPS + grp;
            if (col < d.vdp) {
                const float u = beta * (v_s[col] - g * r[c]);
                if (sub == 0) o_s[col] = fmaf(g, r[DT_CP + c], kq * u);
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (sub + i * LPC < nv)
                        *(reinterpret_cast<float4*>(S + (size_t)col * d.dimp) + sub + i * LPC) =
                            make_float4(fmaf(g, s[c][i].x, k[i].x * u), fmaf(g, s[c][i].y, k[i].y * u), fmaf(g, s[c][i].z, k[i].z * u),
                                        fmaf(g, s[c][i].w, k[i].w * u));
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = lane; c < d.vdp; c += 32) ss = fmaf(o_s[c], o_s[c], ss);
    const float rn = 1.0f / sqrtf(warp_sum(ss) / (float)d.vdim + d.eps);
    for (int c = tid; c < d.vdp; c += DT_THREADS)
        Store<T>::put(a.out + (size_t)m * a.ldo + h * d.vdp + c,
                      o_s[c] * rn * __ldg(a.w.norm + c) * Store<T>::ld(a.gate + (size_t)m * a.ldgate + h * d.vdp + c));
}

}  // namespace vuib
