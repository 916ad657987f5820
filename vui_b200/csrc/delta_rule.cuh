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
//   many rows       k_delta_rows (convolution, unit norms, gates), then k_delta_scan (token by token) or the chunked form,
//                   then k_delta_gate (output norm and gate, the ring's new rows).
#pragma once
#include "lm_kernels.cuh"

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
            if (lane + 32 * j < d.dimp) out[i * d.dimp + lane + 32 * j] = v[j] * r;
    }
    for (int c = 2 * d.G * d.dimp + threadIdx.x; c < d.C; c += LM_THREADS) out[c] = delta_conv(d, a.w, raw, a.ldraw, ring, pos, back, c);
    for (int h = threadIdx.x; h < d.H; h += LM_THREADS) a.gates[(size_t)m * d.H + h] = delta_gates(d, a.w, raw, h);
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

template <class T>
static __global__ void __launch_bounds__(LM_THREADS) k_delta_gate(DeltaGateArgs<T> a) {
    pdl_trigger();
    pdl_wait();
    const DeltaShape& d = a.d;
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    constexpr int P = DR_MAX_VDIM / 64;
    for (int h = warp; h < d.H; h += LM_WARPS) {
        const float* o = a.o + ((size_t)m * d.H + h) * d.vdp;
        const T* gt = a.gate + (size_t)m * a.ldgate + h * d.vdp;
        float2 v[P];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const int c = 2 * (lane + 32 * j);
            v[j] = c < d.vdp ? __ldcg(reinterpret_cast<const float2*>(o + c)) : make_float2(0.f, 0.f);
            ss = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, ss));
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)d.vdim + d.eps);
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const int c = 2 * (lane + 32 * j);
            if (c < d.vdp)
                Store<T>::put2(a.out + (size_t)m * a.ldo + h * d.vdp + c, v[j].x * r * __ldg(a.w.norm + c) * Store<T>::ld(gt + c),
                               v[j].y * r * __ldg(a.w.norm + c + 1) * Store<T>::ld(gt + c + 1));
        }
    }
    if (__ldcg(&a.row_ext[m].y) < d.taps) {
        const int pos = __ldcg(a.row_pos + m);
        float* ring = a.st.ring(__ldcg(a.row_slot + m)) + (size_t)(pos % d.taps) * d.C;
        for (int c = threadIdx.x; c < d.C; c += LM_THREADS) ring[c] = __ldcg(a.raw + (size_t)m * a.ldraw + c);
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
