// libvuib200_lm: C ABI over the token-model kernels (see include/vuib200_lm.h).  The host side validates, lays out the
// caller's workspace and enqueues kernels on the caller's stream; it never allocates device memory.
//
// A layer starts with [norms + every projection of x] and ends with [output + MLP down, residual]: two weight-streaming
// launches for up to LM_FEW_ROWS rows, a norm launch and two tcgen05 GEMMs for more.  Between them:
//   latent    [queries, cache append] [attention, value matrix, gate] for few rows; latent rows, tcgen05 GEMM, attention,
//             value matrix for more; a prefill of many rows expands keys and values instead (latent_prefill.cuh)
//   grouped   one launch in a decode step; [rotation, norms, cache append] [attention] otherwise (grouped_attn.cuh)
//   delta     one launch in a decode step; [convolution, unit norms, gates] [recurrence] [norm, gate] otherwise (delta_rule.cuh)
// 32-bit models: fp32 products, and the latent attention's splits merge in a launch of their own.
#include "../../include/vuib200_lm.h"

#include <algorithm>
#include <cstdarg>
#include <cstdio>
#include <cstring>
#include <map>
#include <new>
#include <type_traits>
#include <utility>
#include <vector>

#include "delta_rule.cuh"
#include "grouped_attn.cuh"
#include "host_common.cuh"
#include "latent_attn.cuh"
#include "latent_prefill.cuh"
#include "lm_kernels.cuh"

using namespace vuib;

namespace {

constexpr int LM_FEW_ROWS = 8;         // rows up to which the weight-streaming products run (fp32: 4)
constexpr int LM_FEW_ROWS_F32 = 4;
constexpr int LA_ROW_BLOCK = 512;      // rows of one fp32 attention launch (bounds the split scratch)
constexpr int LA_CTAS = 2 * 148;       // CTAs the key splits are cut to
// CTAs of a streaming product: one per SM, so that the next kernel's fit beside them and request their weights early;
// two for a matrix of which the next kernel's early requests are a small part.
constexpr int LS_CTAS = 148;
constexpr size_t LS_LARGE = (size_t)48 << 20;
constexpr int LM_EXPAND_MIN = 64;      // rows of a call from which a prefill expands keys and values
constexpr size_t LM_MAX_SMEM = 227 * 1024;

struct LmLayout {
    size_t flag, ctl, row_slot, row_pos, row_ext, segs, xsegs, tiles, x, xn, dq, cq, dkv, gate, q, ay, part, ml, olat;
    size_t tc_partial, tc_counters, xkv, xc;
    size_t raw, dx, dg, dout;   // grouped and delta layers: fp32 rows of the input product; delta: k_delta_rows, recurrence
    size_t dw, du, dp;          // delta, chunked: k_delta_solve
    size_t draw_ctr, rep_counts, rep_hist, rep_head, rep_filled;
    size_t total;
    int ldx, ld_dq, ld_dkv, ld_gate, ld_ay, ld_q, ld_raw;
    int x_rows;      // expanded rows the workspace holds
};

struct LmMaps {      // tensor maps of the packed matrices (dtype bf16)
    CUtensorMap w_in, w_q, w_out, w_xq, w_xkv;
};

}  // namespace

struct VuibLm {
    VuibLmConfig cfg;
    std::vector<VuibLmLayer> layer;
    std::vector<VuibLmDims> dims;
    std::vector<VuibLmLayerWeights> w;
    std::vector<LmMaps> maps;
    CUtensorMap map_head;
    VuibLmHeadWeights head;
    std::vector<void*> cache;
    int32_t* seq_lens;
    unsigned char* ws;
    LmLayout lay;
    bool have_w, have_cache, have_ws;
    int R;                 // rows of scratch
    bool recurrent;        // some layer's state is carried from token to token
    int few_rows;          // rows up to which the streaming products run for this model's sizes
    int num_sms;
    unsigned spin_limit;
    int expand_min;
    float* taps;
    long long launches;
    char err[256];
};

namespace {

int32_t fail(VuibLm* e, int32_t code, const char* fmt, ...) {
    if (e) {
        va_list ap;
        va_start(ap, fmt);
        vsnprintf(e->err, sizeof(e->err), fmt, ap);
        va_end(ap);
    }
    return code;
}

#define CK(call)                                                                              \
    do {                                                                                      \
        cudaError_t _err = (call);                                                            \
        if (_err != cudaSuccess)                                                              \
            return fail(e, VUIB_ERR_CUDA, "%s failed: %s", #call, cudaGetErrorString(_err));  \
    } while (0)
#define RC(call)                       \
    do {                               \
        int32_t _rc = (call);          \
        if (_rc != VUIB_OK) return _rc; \
    } while (0)

int up(int v, int m) { return (v + m - 1) / m * m; }

template <class T>
T* wsp(VuibLm* e, size_t off) { return reinterpret_cast<T*>(e->ws + off); }

VuibLmDims layer_dims(const VuibLmConfig& c, const VuibLmLayer& l) {
    VuibLmDims d;
    memset(&d, 0, sizeof(d));
    const bool mlp = l.mlp != VUIB_LM_MLP_NONE, b16 = c.dtype == VUIB_LM_BF16;
    d.k_in = up(c.width, 64);
    d.n_out = up(c.width, 128);
    d.dimp = up(l.dim, 16);
    d.vdp = up(l.vdim, 16);
    if (l.mixer == VUIB_LM_MIX_LATENT) {
        d.rp = up(l.kv_rank, 16);
        d.rotp = up(l.rot_dim, 16);
        d.dp = d.rp + d.rotp;
        d.n_dq = up(l.q_rank, 16);
        d.n_kv = d.n_dq + d.dp;
        d.n_gate = d.n_kv + up(l.heads * l.vdim, 16);
        d.n_mlp = up(d.n_gate, 128);
        d.k_q = up(l.q_rank, 64);
        d.n_q = up(l.heads * d.dp, 128);
        d.off_y = up(l.heads * l.vdim, 64);
        d.x_ok = b16 && latent_prefill_fits(d.dimp + d.rotp, d.vdp);
        d.n_xq = up(l.heads * (d.dimp + d.rotp), 128);
        d.k_kv = up(d.rp, 64);
        d.n_xkv = up(l.heads * (d.dimp + d.vdp), 128);
        d.slot_bytes = (int64_t)c.max_seq * d.dp * (b16 ? 2 : 4);
    } else {
        const bool delta = l.mixer == VUIB_LM_MIX_DELTA;
        d.n_key = (delta ? l.kv_heads : l.heads) * d.dimp;
        d.n_value = d.n_key + l.kv_heads * d.dimp;
        d.n_ab = d.n_value + (delta ? l.heads : l.kv_heads) * d.vdp;
        d.n_raw = d.n_ab + (delta ? up(2 * l.heads, 16) : 0);
        d.n_gate = d.n_raw + (delta ? l.heads * d.vdp : 0);
        d.n_mlp = d.n_gate;
        d.off_y = up(l.heads * d.vdp, 64);
        if (delta) {
            d.off_v = (int64_t)l.heads * d.vdp * d.dimp;
            d.slot_bytes = 4 * (d.off_v + (int64_t)l.taps * d.n_ab);
        } else {
            // the ring: a window (read from a multiple of LA_UNIT on) and the rows of one call, or every position
            const int64_t all = up(c.max_seq, GP_TILE), part = l.window > 0 ? ((int64_t)l.window + LA_UNIT + c.max_prefill_rows + GP_TILE - 1) / GP_TILE * GP_TILE : all;
            d.cap = (int32_t)(part < all ? part : all);
            d.off_v = (int64_t)l.kv_heads * d.cap * d.dimp;
            d.slot_bytes = (d.off_v + (int64_t)l.kv_heads * d.cap * d.vdp) * (b16 ? 2 : 4);
        }
    }
    d.n_in = up(d.n_mlp + (mlp ? (l.mlp == VUIB_LM_MLP_CLAMPED_GLU ? 2 : 1) * l.ff : 0), 128);
    d.k_out = d.off_y + (mlp ? up(l.ff, 64) : 0);
    return d;
}

// Delta layers whose prefill runs in chunks.
bool chunked_delta(const VuibLmConfig& c, const VuibLmDims& d) { return c.dtype == VUIB_LM_BF16 && d.dimp <= DC_MAX_DIM; }

int attn_splits(VuibLm* e, int li, int M) {
    const VuibLmLayer& l = e->layer[li];
    const int units = M * ((l.heads + 15) / 16);
    const int keys = e->cfg.dtype == VUIB_LM_BF16 ? LA_KEYS : LA_KEYS_F32;
    int s = (LA_CTAS + units - 1) / units;
    const int most = (e->cfg.max_seq + keys - 1) / keys;
    if (s > most) s = most;
    if (s > LA_MAX_SPLITS) s = LA_MAX_SPLITS;
    return s < 1 ? 1 : s;
}

void make_layout(VuibLm* e) {
    const VuibLmConfig& c = e->cfg;
    LmLayout& L = e->lay;
    const size_t R = e->R, es = c.dtype == VUIB_LM_BF16 ? 2 : 4;
    size_t off = 0;
    auto take = [&](size_t bytes) { size_t o = off; off = align_up(off + bytes); return o; };
    int dq = 0, cq = 0, dkv = 0, gate = 0, q = 0, ay = 0, xkv = 0, xc = 0, olat = 0, raw = 0, dx = 0, dg = 0, dout = 0, dw = 0;
    int du = 0, dp = 0;
    size_t part = 0, ml = 0;
    for (size_t i = 0; i < e->layer.size(); ++i) {
        const VuibLmLayer& l = e->layer[i];
        const VuibLmDims& d = e->dims[i];
        auto mx = [](int& a, int b) { if (b > a) a = b; };
        mx(ay, d.k_out);
        if (l.mixer != VUIB_LM_MIX_LATENT) {
            mx(raw, d.n_raw);
            mx(gate, d.n_gate - d.n_raw);
            if (l.mixer == VUIB_LM_MIX_GROUPED) {
                mx(q, l.heads * d.dimp);
            } else {
                mx(dx, d.n_ab);
                mx(dg, 2 * l.heads);
                mx(dout, l.heads * d.vdp);
                if (chunked_delta(c, d)) {
                    mx(dw, l.heads * d.dimp);
                    mx(du, l.heads * d.vdp);
                    mx(dp, l.heads * DC_ROWS);
                }
            }
            continue;
        }
        mx(dq, d.n_dq);
        mx(cq, d.k_q);
        mx(dkv, d.dp);
        mx(gate, d.n_gate - d.n_kv);
        mx(q, l.heads * d.dp);
        if (d.x_ok) {
            mx(q, l.heads * (d.dimp + d.rotp));
            mx(xkv, l.heads * (d.dimp + d.vdp));
            mx(xc, d.k_kv);
        }
        mx(olat, l.heads * d.rp);
        for (int m = 1; c.dtype == VUIB_LM_F32 && m <= LA_ROW_BLOCK && m <= (int)R; ++m) {
            const size_t rows = (size_t)m * attn_splits(e, (int)i, m) * l.heads;
            if (rows * d.rp > part) part = rows * d.rp;
            if (rows * 2 > ml) ml = rows * 2;
        }
    }
    L.ldx = up(c.width, 64);
    L.ld_dq = dq;
    L.ld_dkv = dkv;
    L.ld_gate = gate;
    L.ld_ay = ay;
    L.ld_q = q;
    L.ld_raw = raw;
    L.x_rows = xkv ? (int)R + c.max_seq : 0;
    L.flag = take(256);
    L.ctl = take(sizeof(SamplingCtl));
    L.row_slot = take(R * 4);
    L.row_pos = take(R * 4);
    L.row_ext = take(R * 8);
    L.segs = take(R * 16);
    L.xsegs = take(R * 16);
    L.tiles = take(R * 32);
    L.x = take(R * L.ldx * 4);
    L.xn = take(2 * R * L.ldx * es);
    L.dq = take(R * dq * 4);
    L.cq = take(R * cq * es);
    L.dkv = take(R * dkv * 4);
    L.gate = take(R * gate * es);
    L.q = take(R * q * es);
    L.ay = take(R * ay * es);
    L.part = take(part * 4);
    L.ml = take(ml * 4);
    L.olat = take(c.dtype == VUIB_LM_BF16 ? R * olat * 2 : 0);
    L.tc_partial = take(c.dtype == VUIB_LM_BF16 ? tc_partial_bytes(R + L.x_rows) : 0);
    L.tc_counters = take(2 * TC_COUNTERS * 4);
    L.xkv = take((size_t)L.x_rows * xkv * es);
    L.xc = take((size_t)L.x_rows * xc * es);
    L.raw = take(R * raw * 4);
    L.dx = take(R * dx * 4);
    L.dg = take(R * dg * 4);
    L.dout = take(R * dout * 4);
    L.dw = take(R * dw * 4);
    L.du = take(R * du * 4);
    L.dp = take(R * dp * 4);
    L.draw_ctr = take((size_t)c.n_slots * 4);
    L.rep_counts = take((size_t)c.n_slots * c.vocab * 4);
    L.rep_hist = take((size_t)c.n_slots * REP_HIST_MAX * 4);
    L.rep_head = take((size_t)c.n_slots * 4);
    L.rep_filled = take((size_t)c.n_slots * 4);
    L.total = off;
}

// Opts a kernel into its dynamic shared memory, once per device and only upwards.
cudaError_t allow_smem(const void* kern, size_t bytes) {
    static std::mutex mu;
    static std::map<std::pair<int, const void*>, size_t> have;
    int dev = 0;
    cudaError_t err = cudaGetDevice(&dev);
    if (err != cudaSuccess) return err;
    std::lock_guard<std::mutex> lock(mu);
    size_t& h = have[{dev, kern}];
    if (bytes <= 32 * 1024 || bytes <= h) return cudaSuccess;   // static shared memory counts towards the 48 KB default
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (err == cudaSuccess) h = bytes;
    return err;
}

template <class... KArgs, class... Args>
int32_t run_cl(VuibLm* e, void (*kern)(KArgs...), dim3 grid, int cluster, int threads, size_t smem, cudaStream_t s, Args... args) {
    CK(allow_smem(reinterpret_cast<const void*>(kern), smem));
    CK(launch_cl(kern, grid, cluster, threads, smem, s, args...));
    e->launches++;
    return VUIB_OK;
}

template <class... KArgs, class... Args>
int32_t run(VuibLm* e, void (*kern)(KArgs...), dim3 grid, int threads, size_t smem, cudaStream_t s, Args... args) {
    return run_cl(e, kern, grid, 1, threads, smem, s, args...);
}

// ---------------------------------------------------------------------------
// Matrix products
// ---------------------------------------------------------------------------
constexpr size_t LS_MAX_SMEM = 200 * 1024;

// CTAs of a cluster along K for a product whose rows alone do not fill the SMs.
int stream_ck(int n_groups, int K, bool k_parts) {
    int ck = 1;
    if ((size_t)n_groups * 32 * K > LS_LARGE) return 1;
    while (k_parts && ck < 4 && n_groups * ck * 2 <= LS_CTAS && K % (64 * ck) == 0 && K / (2 * ck) >= 256) ck *= 2;
    return ck;
}

template <class Stage>
size_t stream_smem(int rt, int K, int ck) { return (size_t)Stage::TILES * rt * (K / ck + LS_PAD) * 2 + Stage::scratch(rt, K); }

template <int RT, class Stage, class Epi>
int32_t stream_rt(VuibLm* e, const Stage& st, const Epi& ep, const void* W, int K, int M, int n_rows, cudaStream_t s) {
    StreamArgs a;
    a.W = static_cast<const bf16*>(W);
    a.K = K;
    a.M = M;
    a.n_groups = (n_rows + 15) / 16;
    a.ck = stream_ck(a.n_groups, K, Stage::K_PARTS);
    // warps along K: as many as the one wave of CTAs has to spare, two 32-k blocks each at least
    a.kw = 1;
    const int blocks = K / a.ck / 32, wave = (size_t)n_rows * K * 2 > LS_LARGE ? 2 * LS_CTAS : LS_CTAS;
    while (a.kw < LM_WARPS && a.n_groups * a.ck * a.kw * 2 <= wave * LM_WARPS && a.kw * 4 <= blocks) a.kw *= 2;
    const int gpc = LM_WARPS / a.kw, need = (a.n_groups + gpc - 1) / gpc, most = wave / a.ck;
    const int sets = (need + most - 1) / most, ctas = (need + sets - 1) / sets;
    return run_cl(e, k_lm_stream<RT, Stage, Epi>, dim3(ctas * a.ck + (Stage::HAS_EXTRA ? 1 : 0)), a.ck, LM_THREADS,
                  stream_smem<Stage>(RT, K, a.ck), s, st, ep, a);
}

template <int RT, class Stage, class Epi>
int32_t gemv_rt(VuibLm* e, const Stage& st, const Epi& ep, const void* W, int K, int M, int n_pairs, cudaStream_t s) {
    const int nv = K / Store<float>::VEC;
    int wk = 1;   // warps along K: enough CTAs for every SM, at least one vector per lane
    while (wk < LM_WARPS && (n_pairs + LM_WARPS / wk - 1) / (LM_WARPS / wk) < LA_CTAS && 32 * wk < nv) wk *= 2;
    const int per = LM_WARPS / wk, grid = (n_pairs + per - 1) / per + (Stage::HAS_EXTRA ? 1 : 0);
    return run(e, k_lm_gemv<float, RT, Stage, Epi>, dim3(grid), LM_THREADS, Stage::smem(RT, K), s, st, ep,
               static_cast<const float*>(W), K, M, n_pairs, wk);
}

// n_rows weight rows times up to few_rows activation rows.
template <class T, class Stage, class Epi>
int32_t few(VuibLm* e, const Stage& st, const Epi& ep, const void* W, int K, int M, int n_rows, cudaStream_t s) {
    if constexpr (std::is_same<T, bf16>::value) {
        if (M <= 1) return stream_rt<1>(e, st, ep, W, K, M, n_rows, s);
        if (M <= 2) return stream_rt<2>(e, st, ep, W, K, M, n_rows, s);
        if (M <= 4) return stream_rt<4>(e, st, ep, W, K, M, n_rows, s);
        return stream_rt<8>(e, st, ep, W, K, M, n_rows, s);
    } else {
        const int n_pairs = (n_rows + 1) / 2;
        if (M > 2 && Stage::smem(4, K) <= LS_MAX_SMEM) return gemv_rt<4>(e, st, ep, W, K, M, n_pairs, s);
        if (M > 1 && Stage::smem(2, K) <= LS_MAX_SMEM) return gemv_rt<2>(e, st, ep, W, K, M, n_pairs, s);
        return gemv_rt<1>(e, st, ep, W, K, M, n_pairs, s);
    }
}

// Rows up to which `few` fits shared memory in every product of the model (0: not even one).
int few_rows_of(const VuibLm* e) {
    const VuibLmConfig& c = e->cfg;
    const bool b16 = c.dtype == VUIB_LM_BF16;
    for (int rt = b16 ? LM_FEW_ROWS : LM_FEW_ROWS_F32; rt >= 1; rt /= 2) {
        bool ok = true;
        for (size_t i = 0; i < e->dims.size(); ++i) {
            const VuibLmDims& d = e->dims[i];
            const bool latent = e->layer[i].mixer == VUIB_LM_MIX_LATENT;
            size_t most;
            if (b16) {
                most = stream_smem<StageRowsT<bf16>>(rt, d.k_out, stream_ck(up(c.width, 16) / 16, d.k_out, true));
                const size_t in = latent ? stream_smem<StageLayerNorm2<bf16>>(rt, d.k_in, 1) : stream_smem<StageRms<bf16>>(rt, d.k_in, 1);
                const size_t q = latent ? stream_smem<StageLatentQ<bf16>>(rt, d.k_q, 1) : 0;
                most = std::max(most, std::max(in, q));
            } else {   // one row at a time will do
                most = std::max(StageRowsT<float>::smem(1, d.k_out), StageRowsT<float>::smem(1, d.k_q));
                most = std::max(most, latent ? StageLayerNorm2<float>::smem(1, d.k_in) : StageRms<float>::smem(1, d.k_in));
            }
            ok = ok && most <= LS_MAX_SMEM;
        }
        if (ok) return rt;
    }
    return 0;
}

// Rows [row_off, row_off + n_rows) of W (n_rows a multiple of 128) times M rows of X; weight rows >= n_split (counted
// from row_off) take their rows of X x_off rows further down.
template <class T, class Epi>
int32_t gemm(VuibLm* e, const CUtensorMap& map, const void* W, const T* X, int ldx, int K, int M, int n_rows, const Epi& ep,
             cudaStream_t s, int n_split = 1 << 30, int x_off = 0) {
    if constexpr (std::is_same<T, bf16>::value) {
        const TcCtx cx{wsp<float>(e, e->lay.tc_partial), wsp<int32_t>(e, e->lay.tc_counters), wsp<int32_t>(e, e->lay.flag),
                       nullptr, &e->num_sms, e->spin_limit, &e->launches};
        CK(tc_gemm_launch(cx, map, map, X, ldx, M, K, n_rows, 0, typename TcForm<Epi>::type{ep}, s,
                          n_split < n_rows ? n_split / TC_TILE_N : 1 << 30, n_split < n_rows ? x_off : 0));
        return VUIB_OK;
    } else {
        return run(e, k_gemm_f32<Epi>, dim3(n_rows / 64, (M + 63) / 64), 256, 0, s, X, ldx, static_cast<const float*>(W), K, M,
                   n_split, x_off, ep);
    }
}

// ---------------------------------------------------------------------------
// Attention
// ---------------------------------------------------------------------------
LatentAttnArgs attn_args(VuibLm* e, int li) {
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const LmLayout& L = e->lay;
    LatentAttnArgs a;
    memset(&a, 0, sizeof(a));
    a.q = e->ws + L.q;
    a.cache = e->cache[li];
    a.row_slot = wsp<int32_t>(e, L.row_slot);
    a.row_pos = wsp<int32_t>(e, L.row_pos);
    a.H = l.heads;
    a.Rp = d.rp;
    a.Dp = d.dp;
    a.max_seq = e->cfg.max_seq;
    a.n_slots = e->cfg.n_slots;
    a.scale = l.scale;
    a.row_vecs = FastDiv(d.dp / 8);
    a.w_vecs = FastDiv(d.rp / 8);
    return a;
}

template <bool FUSE_V>
int32_t latent_attn_nt(VuibLm* e, const LatentAttnArgs& a, int CL, int M, cudaStream_t s) {
    const dim3 grid(CL * ((a.H + 15) / 16), M);
    const size_t sm = latent_attn_smem(a.Dp, a.Rp, a.keys, a.nbuf, FUSE_V ? 16 / CL : 0, FUSE_V ? 16 / CL * a.vdim : 0);
    if (a.Rp <= 128) return run_cl(e, k_latent_attn<2, FUSE_V>, grid, CL, LM_THREADS, sm, s, a, CL);
    if (a.Rp <= 256) return run_cl(e, k_latent_attn<4, FUSE_V>, grid, CL, LM_THREADS, sm, s, a, CL);
    if (a.Rp <= 512) return run_cl(e, k_latent_attn<8, FUSE_V>, grid, CL, LM_THREADS, sm, s, a, CL);
    return run_cl(e, k_latent_attn<16, FUSE_V>, grid, CL, LM_THREADS, sm, s, a, CL);
}

int32_t absorbed_attention_bf16(VuibLm* e, int li, int M, cudaStream_t s) {
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const LmLayout& L = e->lay;
    LatentAttnArgs a = attn_args(e, li);
    // splits of a row's keys: one wave of CTAs, no more than the cache has tiles
    const int units = M * ((l.heads + 15) / 16);
    int CL = 1;
    while (CL < LA_MAX_CL && units * CL * 2 <= LA_CTAS && CL * LA_KEYS / 2 < e->cfg.max_seq) CL *= 2;
    a.keys = LA_KEYS;
    while (a.keys > 32 && latent_attn_smem(d.dp, d.rp, a.keys, 1) > LM_MAX_SMEM) a.keys /= 2;
    const bool fuse = M <= LM_FEW_ROWS && latent_attn_smem(d.dp, d.rp, a.keys, 1, 16 / CL, 16 / CL * l.vdim) <= LM_MAX_SMEM;
    // a second key tile in flight where it costs no resident CTA
    a.nbuf = latent_attn_smem(d.dp, d.rp, a.keys, 2, fuse ? 16 / CL : 0, fuse ? 16 / CL * l.vdim : 0) <= (fuse ? LM_MAX_SMEM : LM_MAX_SMEM / 2) ? 2 : 1;
    a.wuv = static_cast<const bf16*>(e->w[li].w_uv);
    a.gate = wsp<bf16>(e, L.gate);
    a.ldgate = L.ld_gate;
    a.vdim = l.vdim;
    a.ldo = L.ld_ay;
    if (fuse) {
        a.out = wsp<bf16>(e, L.ay);
        return latent_attn_nt<true>(e, a, CL, M, s);
    }
    a.out = wsp<bf16>(e, L.olat);
    RC(latent_attn_nt<false>(e, a, CL, M, s));
    const LatentValueArgs v{a.wuv, wsp<bf16>(e, L.olat), a.gate, L.ld_gate, wsp<bf16>(e, L.ay), L.ld_ay, l.heads, d.rp, l.vdim, M};
    return run(e, k_latent_value, dim3(l.heads, (l.vdim + 63) / 64, (M + 8 * LV_TILES - 1) / (8 * LV_TILES)), 128, 0, s, v);
}

int32_t absorbed_attention_f32(VuibLm* e, int li, int M, cudaStream_t s) {
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const LmLayout& L = e->lay;
    for (int m0 = 0; m0 < M; m0 += LA_ROW_BLOCK) {
        const int m = M - m0 < LA_ROW_BLOCK ? M - m0 : LA_ROW_BLOCK;
        LatentAttnArgs a = attn_args(e, li);
        a.q = wsp<float>(e, L.q) + (size_t)m0 * l.heads * d.dp;
        a.row_slot += m0;
        a.row_pos += m0;
        a.part = wsp<float>(e, L.part);
        a.ml = wsp<float>(e, L.ml);
        a.S = attn_splits(e, li, m);
        a.nbuf = 1;
        const int nc = d.rp <= 128 ? 8 : 32;
        a.col_blocks = (d.rp + nc * 16 - 1) / (nc * 16);
        const dim3 grid(a.S, (l.heads + 15) / 16 * a.col_blocks, m);
        const size_t sm = latent_attn_f32_smem(d.dp);
        if (nc == 8) RC(run(e, k_latent_attn_f32<8>, grid, LM_THREADS, sm, s, a));
        else RC(run(e, k_latent_attn_f32<32>, grid, LM_THREADS, sm, s, a));
        LatentOutArgs o;
        o.part = a.part;
        o.ml = a.ml;
        o.row_pos = a.row_pos;
        o.wuv = e->w[li].w_uv;
        o.gate = wsp<float>(e, L.gate) + (size_t)m0 * L.ld_gate;
        o.ldgate = L.ld_gate;
        o.out = wsp<float>(e, L.ay) + (size_t)m0 * L.ld_ay;
        o.ldo = L.ld_ay;
        o.H = l.heads;
        o.Rp = d.rp;
        o.vdim = l.vdim;
        o.S = a.S;
        o.keys = LA_KEYS_F32;
        o.M = m;
        const int rt = m == 1 ? 1 : 4, rows = (m + rt - 1) / rt;
        int vs = (148 + l.heads * rows - 1) / (l.heads * rows);   // slices of the value dimensions, >= 8 each
        if (vs > (l.vdim + 7) / 8) vs = (l.vdim + 7) / 8;
        const dim3 og(l.heads, rows, vs);
        if (rt == 1) RC(run(e, k_latent_out<float, 1>, og, LM_THREADS, (size_t)d.rp * 4, s, o));
        else RC(run(e, k_latent_out<float, 4>, og, LM_THREADS, (size_t)4 * d.rp * 4, s, o));
    }
    return VUIB_OK;
}

template <class T>
int32_t absorbed_attention(VuibLm* e, int li, int M, cudaStream_t s) {
    if constexpr (std::is_same<T, bf16>::value) return absorbed_attention_bf16(e, li, M, s);
    else return absorbed_attention_f32(e, li, M, s);
}

struct ExpandGroup {   // sequences of a prefill whose keys are expanded together
    int tile0, n_tiles, seg0, n_segs, rows;
};

int32_t expanded_attention(VuibLm* e, int li, const ExpandGroup& g, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const LmLayout& L = e->lay;
    const bf16* cache = static_cast<const bf16*>(e->cache[li]);
    bf16* xc = wsp<bf16>(e, L.xc);
    bf16* xkv = wsp<bf16>(e, L.xkv);
    const int n_x = l.heads * (d.dimp + d.vdp);
    const LatentGatherArgs ga{cache, wsp<int4>(e, L.xsegs) + g.seg0, g.n_segs, g.rows, xc, d.k_kv, d.rp, d.dp, c.max_seq};
    RC(run(e, k_latent_gather, dim3((g.rows + 7) / 8), 256, 0, s, ga));
    RC(gemm<bf16>(e, e->maps[li].w_xkv, e->w[li].w_xkv, xc, d.k_kv, d.k_kv, g.rows, d.n_xkv, EpRows<bf16>{xkv, n_x, n_x}, s));
    LatentPrefillArgs a;
    a.q = wsp<bf16>(e, L.q);
    a.xkv = xkv;
    a.ldx = n_x;
    a.cache = cache;
    a.tiles = wsp<int4>(e, L.tiles) + 2 * g.tile0;
    a.gate = wsp<bf16>(e, L.gate);
    a.ldgate = L.ld_gate;
    a.out = wsp<bf16>(e, L.ay);
    a.ldo = L.ld_ay;
    a.H = l.heads;
    a.dimp = d.dimp;
    a.rotp = d.rotp;
    a.vdim = l.vdim;
    a.vdp = d.vdp;
    a.Rp = d.rp;
    a.Dp = d.dp;
    a.max_seq = c.max_seq;
    a.scale = l.scale;
    a.key_vecs = FastDiv((d.dimp + d.rotp + d.vdp) / 8);
    const int qk = d.dimp + d.rotp;
    const size_t sm = latent_prefill_smem(qk, d.vdp);
    const dim3 grid(g.n_tiles, l.heads);
    if (d.vdp <= 64) {
        if (qk <= 96) return run(e, k_latent_prefill<6, 4>, grid, 128, sm, s, a);
        if (qk <= 192) return run(e, k_latent_prefill<12, 4>, grid, 128, sm, s, a);
        return run(e, k_latent_prefill<16, 4>, grid, 128, sm, s, a);
    }
    if (qk <= 96) return run(e, k_latent_prefill<6, 8>, grid, 128, sm, s, a);
    if (qk <= 192) return run(e, k_latent_prefill<12, 8>, grid, 128, sm, s, a);
    return run(e, k_latent_prefill<16, 8>, grid, 128, sm, s, a);
}

// ---------------------------------------------------------------------------
// What a pass over the layers knows of its rows besides what is in the workspace.
// ---------------------------------------------------------------------------
struct Pass {
    int M;
    bool step;         // a decode step: every row one token of a slot of its own
    int n_segs;        // portions of a prefill
    int n_tiles;       // query tiles of a prefill that runs the mixers' prefill forms (0: it does not)
    const std::vector<ExpandGroup>* expand;
    bool few;          // the weight-streaming products run
};

// The input product of a layer: norm (few rows: in the staging) and every matrix that reads x.
template <class T, class Stage, class Epi>
int32_t product_in(VuibLm* e, int li, const Pass& ps, const Stage& st, const Epi& ep, NormVec n1, NormVec n2, int n_split, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    const VuibLmDims& d = e->dims[li];
    if (ps.few) return few<T>(e, st, ep, e->w[li].w_in, d.k_in, ps.M, d.n_in, s);
    T* xn = wsp<T>(e, L.xn);
    T* xn2 = n2.w ? xn + (size_t)e->R * L.ldx : nullptr;
    auto norm = c.block == VUIB_LM_BLOCK_LN2 ? k_norm_rows<T, true> : k_norm_rows<T, false>;
    RC(run(e, norm, dim3(ps.M), 128, 0, s, wsp<float>(e, L.x), L.ldx, c.width, c.norm_eps, n1, xn, n2, xn2, L.ldx, nullptr, nullptr,
           nullptr, nullptr));
    return gemm<T>(e, e->maps[li].w_in, e->w[li].w_in, xn, L.ldx, d.k_in, ps.M, d.n_in, ep, s, n_split, e->R);
}

// x += W_out [mixer | MLP] (+ bias)
template <class T>
int32_t product_out(VuibLm* e, int li, const Pass& ps, cudaStream_t s) {
    const LmLayout& L = e->lay;
    const VuibLmDims& d = e->dims[li];
    const T* ay = wsp<T>(e, L.ay);
    const EpAddResidual er{wsp<float>(e, L.x), L.ldx, e->cfg.width, e->w[li].b_out};
    if (ps.few) return few<T>(e, StageRowsT<T>{ay, L.ld_ay}, er, e->w[li].w_out, d.k_out, ps.M, e->cfg.width, s);
    return gemm<T>(e, e->maps[li].w_out, e->w[li].w_out, ay, L.ld_ay, d.k_out, ps.M, d.n_out, er, s);
}

template <class T>
int32_t latent_layer(VuibLm* e, int li, const Pass& ps, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const VuibLmLayerWeights& w = e->w[li];
    const LmMaps& mp = e->maps[li];
    const int M = ps.M;
    float* x = wsp<float>(e, L.x);
    const bool ex = ps.expand && d.x_ok && !ps.few;
    const NormVec n1{w.norm1_w, w.norm1_b}, n2{w.norm2_w, w.norm2_b};
    const float2* trig = reinterpret_cast<const float2*>(w.trig);
    EpBlockIn<T> ei;
    ei.n_dq = d.n_dq;
    ei.n_kv = d.n_kv;
    ei.n_gate = d.n_gate;
    ei.n_mlp = d.n_mlp;
    ei.ff = l.mlp == VUIB_LM_MLP_NONE ? 0 : l.ff;
    ei.dq = wsp<float>(e, L.dq);
    ei.lddq = L.ld_dq;
    ei.dkv = wsp<float>(e, L.dkv);
    ei.lddkv = d.dp;
    ei.gate = wsp<T>(e, L.gate);
    ei.ldgate = L.ld_gate;
    ei.act = wsp<T>(e, L.ay) + d.off_y;
    ei.ldact = L.ld_ay;
    ei.limit = l.mlp_limit;
    ei.slope = l.mlp_slope;
    ei.shift = l.mlp_shift;
    const LatentRow lat{wsp<float>(e, L.dkv), w.kv_norm, c.norm_eps, l.kv_rank, d.rp, l.rot_dim, l.rot_dims, d.dp, trig,
                        e->cache[li], wsp<int32_t>(e, L.row_slot), wsp<int32_t>(e, L.row_pos), c.max_seq};
    const int head_rows = ex ? d.dimp + d.rotp : d.dp;
    const EpRotatedQ<T> eq{wsp<T>(e, L.q), l.heads * head_rows, head_rows, head_rows - d.rotp, l.rot_dims, trig,
                           wsp<int32_t>(e, L.row_pos)};
    const StageLayerNorm2<T> sn{x, L.ldx, c.width, c.norm_eps, n1, n2, d.n_mlp, nullptr};
    RC(product_in<T>(e, li, ps, sn, ei, n1, n2, d.n_mlp, s));
    if (ps.few) {
        const StageLatentQ<T> sq{{wsp<float>(e, L.dq), L.ld_dq, l.q_rank, c.norm_eps, w.q_norm}, lat};
        RC(few<T>(e, sq, eq, w.w_q, d.k_q, M, l.heads * d.dp, s));
    } else {
        RC(run(e, k_latent_rows<T>, dim3(M), 128, 0, s, lat, wsp<float>(e, L.dq), L.ld_dq, l.q_rank, w.q_norm,
               wsp<T>(e, L.cq), d.k_q));
        RC(gemm<T>(e, ex ? mp.w_xq : mp.w_q, ex ? w.w_xq : w.w_q, wsp<T>(e, L.cq), d.k_q, d.k_q, M, ex ? d.n_xq : d.n_q, eq, s));
    }
    if (ex) {
        if constexpr (std::is_same<T, bf16>::value) {
            for (const ExpandGroup& g : *ps.expand) RC(expanded_attention(e, li, g, s));
        }
    } else {
        RC(absorbed_attention<T>(e, li, M, s));
    }
    return product_out<T>(e, li, ps, s);
}

// The input product of the layers with one RMS norm.
template <class T>
int32_t mix_in(VuibLm* e, int li, const Pass& ps, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const NormVec n1{e->w[li].norm1_w, nullptr};
    const EpMixIn<T> ei{d.n_raw, d.n_gate, d.n_mlp, l.mlp == VUIB_LM_MLP_NONE ? 0 : l.ff, e->w[li].b_in, wsp<float>(e, L.raw), L.ld_raw,
                        wsp<T>(e, L.gate), L.ld_gate, wsp<T>(e, L.ay) + d.off_y, L.ld_ay};
    const StageRms<T> st{wsp<float>(e, L.x), L.ldx, c.width, c.norm_eps, n1.w};
    return product_in<T>(e, li, ps, st, ei, n1, NormVec{nullptr, nullptr}, 1 << 30, s);
}

template <bool OWN>
int32_t grouped_rows_bf16(VuibLm* e, int li, const QkRowsArgs& r, int M, cudaStream_t s) {
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    GroupedAttnArgs a;
    memset(&a, 0, sizeof(a));
    a.r = r;
    a.q = static_cast<const bf16*>(r.q);
    a.out = wsp<bf16>(e, e->lay.ay);
    a.ldo = e->lay.ld_ay;
    a.window = l.window > 0 ? l.window : e->cfg.max_seq;
    a.max_seq = e->cfg.max_seq;
    a.n_slots = e->cfg.n_slots;
    a.hpg = l.heads / l.kv_heads;
    a.hgroups = (a.hpg + 15) / 16;
    a.scale = l.scale;
    a.softcap = l.softcap;
    a.k_vecs = FastDiv(d.dimp / 8);
    a.v_vecs = FastDiv(d.vdp / 8);
    const int units = M * l.kv_heads * a.hgroups, seen = std::min(a.window, a.max_seq);
    int CL = 1;
    while (CL < LA_MAX_CL && units * CL * 2 <= LA_CTAS && CL * LA_KEYS / 2 < seen) CL *= 2;
    a.keys = LA_KEYS;
    while (a.keys > 32 && (grouped_attn_smem(d.dimp, d.vdp, a.keys, 1) > LM_MAX_SMEM || a.keys / 2 * CL >= seen + 16)) a.keys /= 2;
    // a second key tile in flight where a split has more than one and it costs no resident CTA
    a.nbuf = a.keys * CL < seen + 16 && grouped_attn_smem(d.dimp, d.vdp, a.keys, 2) <= LM_MAX_SMEM / 2 ? 2 : 1;
    const dim3 grid(CL * a.hgroups * l.kv_heads, M);
    const size_t sm = grouped_attn_smem(d.dimp, d.vdp, a.keys, a.nbuf);
    if (d.vdp <= 128) return run_cl(e, k_grouped_attn<2, OWN>, grid, CL, LM_THREADS, sm, s, a, CL);
    return run_cl(e, k_grouped_attn<4, OWN>, grid, CL, LM_THREADS, sm, s, a, CL);
}

template <int KS>
int32_t grouped_tiles(VuibLm* e, const GroupedPrefillArgs& a, int n_tiles, cudaStream_t s) {
    const dim3 grid(n_tiles, a.H);
    const size_t sm = grouped_prefill_smem(a.c.dimp, a.c.vdp);
    if (a.c.vdp <= 64) return run(e, k_grouped_prefill<KS, 4>, grid, 128, sm, s, a);
    if (a.c.vdp <= 128) return run(e, k_grouped_prefill<KS, 8>, grid, 128, sm, s, a);
    return run(e, k_grouped_prefill<KS, 16>, grid, 128, sm, s, a);
}

template <class T>
int32_t qk_rows(VuibLm* e, const QkRowsArgs& r, int M, cudaStream_t s) {
    const int p = r.c.dimp <= 64 ? 1 : r.c.dimp <= 128 ? 2 : 4, u = 8 / p;
    const dim3 grid((M * qk_groups(r.H, r.G, r.c.vdp, p, u) + LM_WARPS - 1) / LM_WARPS);
    if (p == 1) return run(e, k_qk_rows<T, 1, 8>, grid, LM_THREADS, 0, s, r, M);
    if (p == 2) return run(e, k_qk_rows<T, 2, 4>, grid, LM_THREADS, 0, s, r, M);
    return run(e, k_qk_rows<T, 4, 2>, grid, LM_THREADS, 0, s, r, M);
}

template <class T>
int32_t grouped_layer(VuibLm* e, int li, const Pass& ps, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    RC(mix_in<T>(e, li, ps, s));
    QkRowsArgs r;
    memset(&r, 0, sizeof(r));
    r.raw = wsp<float>(e, L.raw);
    r.ldraw = L.ld_raw;
    r.n_k = d.n_key;
    r.n_v = d.n_value;
    r.q = wsp<T>(e, L.q);
    r.c = GroupedCache{e->cache[li], (size_t)d.slot_bytes / sizeof(T), (size_t)d.off_v, d.cap, d.dimp, d.vdp};
    r.h = QkHead{reinterpret_cast<const float2*>(e->w[li].trig), l.dim, d.dimp, l.rot_dims, c.norm_eps, l.qk_norm};
    r.row_slot = wsp<int32_t>(e, L.row_slot);
    r.row_pos = wsp<int32_t>(e, L.row_pos);
    r.H = l.heads;
    r.G = l.kv_heads;
    const int window = l.window > 0 ? l.window : c.max_seq, hpg = l.heads / l.kv_heads;
    if constexpr (std::is_same<T, bf16>::value) {
        if (ps.step) {
            RC(grouped_rows_bf16<true>(e, li, r, ps.M, s));
        } else {
            RC(qk_rows<T>(e, r, ps.M, s));
            if (ps.n_tiles) {
                const GroupedPrefillArgs a{static_cast<const bf16*>(r.q), r.c, wsp<int4>(e, L.tiles), wsp<bf16>(e, L.ay), L.ld_ay, l.heads,
                                           hpg, window, l.scale, l.softcap, FastDiv((d.dimp + d.vdp) / 8)};
                if (d.dimp <= 64) RC(grouped_tiles<4>(e, a, ps.n_tiles, s));
                else if (d.dimp <= 128) RC(grouped_tiles<8>(e, a, ps.n_tiles, s));
                else RC(grouped_tiles<16>(e, a, ps.n_tiles, s));
            } else {
                RC(grouped_rows_bf16<false>(e, li, r, ps.M, s));
            }
        }
    } else {
        RC(qk_rows<T>(e, r, ps.M, s));
        const GroupedAttnF32Args a{static_cast<const float*>(r.q), r.c, r.row_slot, r.row_pos, wsp<float>(e, L.ay), L.ld_ay, l.heads, hpg,
                                   window, l.scale, l.softcap};
        RC(run(e, k_grouped_attn_f32, dim3(ps.M, l.heads), LM_THREADS, 0, s, a));
    }
    return product_out<T>(e, li, ps, s);
}

template <class T>
int32_t delta_layer(VuibLm* e, int li, const Pass& ps, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    const VuibLmLayer& l = e->layer[li];
    const VuibLmDims& d = e->dims[li];
    const VuibLmLayerWeights& w = e->w[li];
    RC(mix_in<T>(e, li, ps, s));
    const DeltaShape ds{l.heads, l.kv_heads, l.dim, d.dimp, l.vdim, d.vdp, l.taps, d.n_ab, d.n_ab, l.scale, l.unit_eps, c.norm_eps};
    const DeltaWeights dw{w.conv, w.neg_a, w.dt_bias, w.head_norm};
    const DeltaState st{static_cast<float*>(e->cache[li]), (size_t)d.slot_bytes / 4, (size_t)d.off_v};
    const int32_t *row_slot = wsp<int32_t>(e, L.row_slot), *row_pos = wsp<int32_t>(e, L.row_pos);
    const int2* row_ext = wsp<int2>(e, L.row_ext);
    const DeltaGateArgs<T> ga{ds, dw, st, wsp<float>(e, L.raw), L.ld_raw, wsp<float>(e, L.dout), wsp<T>(e, L.gate), L.ld_gate, wsp<T>(e, L.ay),
                              L.ld_ay, row_slot, row_pos, row_ext};
    if (ps.step) {
        const dim3 grid(l.heads, ps.M);
        if (d.dimp <= 64) RC(run(e, k_delta_step<T, 16, 1>, grid, DT_THREADS, 0, s, ga));
        else if (d.dimp <= 128) RC(run(e, k_delta_step<T, 32, 1>, grid, DT_THREADS, 0, s, ga));
        else RC(run(e, k_delta_step<T, 32, 2>, grid, DT_THREADS, 0, s, ga));
    } else {
        const DeltaRowsArgs ra{ds, dw, st, ga.raw, ga.ldraw, wsp<float>(e, L.dx), wsp<float2>(e, L.dg), row_slot, row_pos, row_ext};
        const bool chunks = ps.n_tiles && chunked_delta(c, d), tile = d.dimp <= 128 && l.taps <= DR_TAPS;
        const dim3 tiles((ps.M + DR_ROWS - 1) / DR_ROWS, (2 * l.kv_heads + (l.heads * d.vdp + 127) / 128 + LM_WARPS - 1) / LM_WARPS);
        if (tile && chunks) RC(run(e, k_delta_rows_tile<true>, tiles, LM_THREADS, 0, s, ra, ps.M));
        else if (tile) RC(run(e, k_delta_rows_tile<false>, tiles, LM_THREADS, 0, s, ra, ps.M));
        else if (chunks) RC(run(e, k_delta_rows<true>, dim3(ps.M), LM_THREADS, 0, s, ra));
        else RC(run(e, k_delta_rows<false>, dim3(ps.M), LM_THREADS, 0, s, ra));
        if (chunks) {
            const DeltaChunkArgs ca{ds, st, ra.out, ra.gates, wsp<int4>(e, L.tiles), wsp<int4>(e, L.segs), wsp<bf16>(e, L.dw), wsp<float>(e, L.du),
                                    wsp<bf16>(e, L.dp), wsp<float>(e, L.dout), FastDiv(d.dimp / 4)};
            RC(run(e, k_delta_solve, dim3(ps.n_tiles, l.heads), LM_THREADS, delta_solve_smem(d.dimp), s, ca));
            const int units = ps.n_segs * l.heads;
            if (units * ((d.vdp + 63) / 64) >= LS_CTAS)
                RC(run(e, k_delta_chunks<64>, dim3(ps.n_segs, l.heads, (d.vdp + 63) / 64), LM_THREADS, delta_chunks_smem<64>(d.dimp), s, ca));
            else if (units * ((d.vdp + 31) / 32) >= LS_CTAS)
                RC(run(e, k_delta_chunks<32>, dim3(ps.n_segs, l.heads, (d.vdp + 31) / 32), LM_THREADS, delta_chunks_smem<32>(d.dimp), s, ca));
            else
                RC(run(e, k_delta_chunks<16>, dim3(ps.n_segs, l.heads, d.vdp / 16), LM_THREADS, delta_chunks_smem<16>(d.dimp), s, ca));
        } else {
            const DeltaScanArgs sa{ds, st, ra.out, ra.gates, wsp<int4>(e, L.segs), wsp<float>(e, L.dout)};
            const int lpc = d.dimp <= 64 ? 16 : 32, cols = DS_THREADS / lpc * DS_CP;
            const dim3 grid(ps.n_segs, l.heads, (d.vdp + cols - 1) / cols);
            if (d.dimp <= 64) RC(run(e, k_delta_scan<16, 1>, grid, DS_THREADS, 0, s, sa));
            else if (d.dimp <= 128) RC(run(e, k_delta_scan<32, 1>, grid, DS_THREADS, 0, s, sa));
            else RC(run(e, k_delta_scan<32, 2>, grid, DS_THREADS, 0, s, sa));
        }
        const int items = ps.M * l.heads;
        if (d.vdp <= 128) RC(run(e, k_delta_gate<T, 1, 4>, dim3((items + 4 * LM_WARPS - 1) / (4 * LM_WARPS)), LM_THREADS, 0, s, ga, ps.M));
        else RC(run(e, k_delta_gate<T, 4, 1>, dim3((items + LM_WARPS - 1) / LM_WARPS), LM_THREADS, 0, s, ga, ps.M));
    }
    return product_out<T>(e, li, ps, s);
}

// One pass over the layers for the rows whose x, slots and positions are in the workspace.
template <class T>
int32_t run_layers(VuibLm* e, Pass ps, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    ps.few = ps.M <= e->few_rows;
    for (int li = 0; li < c.n_layers; ++li) {
        switch (e->layer[li].mixer) {
            case VUIB_LM_MIX_LATENT: RC(latent_layer<T>(e, li, ps, s)); break;
            case VUIB_LM_MIX_GROUPED: RC(grouped_layer<T>(e, li, ps, s)); break;
            default: RC(delta_layer<T>(e, li, ps, s)); break;
        }
        if (e->taps)
            CK(cudaMemcpy2DAsync(e->taps + (size_t)li * e->R * c.width, (size_t)c.width * 4, wsp<float>(e, L.x), (size_t)L.ldx * 4,
                                 (size_t)c.width * 4, ps.M, cudaMemcpyDeviceToDevice, s));
    }
    return VUIB_OK;
}

// Final norm of M rows of x (gathered when rows is given) and logits.
template <class T>
int32_t run_head(VuibLm* e, int M, const int32_t* rows, const int32_t* row_slot, const int32_t* seq_inc, int32_t* seq_lens,
                 float* logits, cudaStream_t s) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    T* xn = wsp<T>(e, L.xn);
    const bool ln = c.block == VUIB_LM_BLOCK_LN2;
    auto norm = ln ? k_norm_rows<T, true> : k_norm_rows<T, false>;
    RC(run(e, norm, dim3(M), 128, 0, s, wsp<float>(e, L.x), L.ldx, c.width, c.norm_eps, NormVec{e->head.final_w, ln ? e->head.final_b : nullptr},
           xn, NormVec{nullptr, nullptr}, static_cast<T*>(nullptr), L.ldx, rows, row_slot, seq_inc, seq_lens));
    const EpLogitsF32 el{logits, c.vocab, c.logit_scale};
    if (M <= e->few_rows) return few<T>(e, StageRowsT<T>{xn, L.ldx}, el, e->head.head, L.ldx, M, c.vocab, s);
    return gemm<T>(e, e->map_head, e->head.head, xn, L.ldx, L.ldx, M, up(c.vocab, 128), el, s);
}

int32_t ready(VuibLm* e) {
    if (!e) return VUIB_ERR_NULL;
    if (!(e->have_w && e->have_cache && e->have_ws))
        return fail(e, VUIB_ERR_UNBOUND, "bind weights, cache and workspace first");
    return VUIB_OK;
}

EmbedArgs embed_args(VuibLm* e, const int64_t* tokens) {
    const VuibLmConfig& c = e->cfg;
    const LmLayout& L = e->lay;
    EmbedArgs a;
    memset(&a, 0, sizeof(a));
    a.tokens = tokens;
    a.table = e->head.embed;
    a.scale = c.embed_scale;
    a.x = wsp<float>(e, L.x);
    a.width = c.width;
    a.ldx = L.ldx;
    a.vocab = c.vocab;
    a.row_slot = wsp<int32_t>(e, L.row_slot);
    a.row_pos = wsp<int32_t>(e, L.row_pos);
    a.row_ext = wsp<int2>(e, L.row_ext);
    a.n_slots = c.n_slots;
    a.max_seq = c.max_seq;
    a.flag = wsp<int32_t>(e, L.flag);
    return a;
}

template <class T>
int32_t prefill(VuibLm* e, const Pass& ps, const int64_t* tokens, int n_want, const int32_t* want, float* logits, cudaStream_t s) {
    EmbedArgs a = embed_args(e, tokens);
    a.segs = wsp<int4>(e, e->lay.segs);
    a.n_segs = ps.n_segs;
    a.seq_lens_out = e->seq_lens;
    RC(run(e, k_lm_embed<T>, dim3(ps.M), 128, 0, s, a));
    RC(run_layers<T>(e, ps, s));
    for (int w0 = 0; w0 < n_want; w0 += e->R) {
        const int n = n_want - w0 < e->R ? n_want - w0 : e->R;
        RC(run_head<T>(e, n, want + w0, nullptr, nullptr, nullptr, logits + (size_t)w0 * e->cfg.vocab, s));
    }
    return VUIB_OK;
}

template <class T>
int32_t decode(VuibLm* e, int B, const int32_t* slots, const int32_t* seq_inc, const int64_t* tokens, float* logits, cudaStream_t s) {
    EmbedArgs a = embed_args(e, tokens);
    a.slots = slots;
    a.seq_lens = e->seq_lens;
    RC(run(e, k_lm_embed<T>, dim3(B), 128, 0, s, a));
    RC(run_layers<T>(e, Pass{B, true, 0, 0, nullptr, false}, s));
    return run_head<T>(e, B, nullptr, wsp<int32_t>(e, e->lay.row_slot), seq_inc, e->seq_lens, logits, s);
}

}  // namespace

// ---------------------------------------------------------------------------
// ABI
// ---------------------------------------------------------------------------
extern "C" int32_t vuib_lm_abi_version(void) { return VUIB_LM_ABI_VERSION; }

extern "C" int32_t vuib_lm_create(const VuibLmConfig* cfg, const VuibLmLayer* layers, VuibLm** out) {
    if (!cfg || !layers || !out) return VUIB_ERR_NULL;
    *out = nullptr;
    const VuibLmConfig& c = *cfg;
    if ((c.dtype != VUIB_LM_BF16 && c.dtype != VUIB_LM_F32) || (c.block != VUIB_LM_BLOCK_LN2 && c.block != VUIB_LM_BLOCK_RMS)) return VUIB_ERR_SHAPE;
    if (c.vocab < 1 || c.width < 1 || c.n_layers < 1 || c.n_layers > VUIB_LM_MAX_LAYERS || !(c.norm_eps >= 0.f)) return VUIB_ERR_SHAPE;
    if (c.n_slots < 1 || c.max_seq < 1 || c.max_rows < 1 || c.max_rows > 65535 || c.max_prefill_rows < 1) return VUIB_ERR_RANGE;
    for (int i = 0; i < c.n_layers; ++i) {
        const VuibLmLayer& l = layers[i];
        if (l.mlp != VUIB_LM_MLP_NONE && l.ff < 1) return VUIB_ERR_SHAPE;
        if (l.heads < 1 || l.dim < 0 || l.vdim < 1) return VUIB_ERR_SHAPE;
        if (c.block == VUIB_LM_BLOCK_LN2) {
            if (l.mixer != VUIB_LM_MIX_LATENT || (l.mlp != VUIB_LM_MLP_NONE && l.mlp != VUIB_LM_MLP_CLAMPED_GLU)) return VUIB_ERR_SHAPE;
            if (l.rot_dim < 0 || l.dim + l.rot_dim < 1 || l.kv_rank < 1 || l.q_rank < 1 || l.rot_dims < 0 || l.rot_dims > l.rot_dim ||
                l.rot_dims % 2)
                return VUIB_ERR_SHAPE;
            const VuibLmDims d = layer_dims(c, l);
            if (c.dtype == VUIB_LM_BF16 ? d.rp > 1024 || latent_attn_smem(d.dp, d.rp, 32, 1) > LM_MAX_SMEM
                                        : latent_attn_f32_smem(d.dp) > LM_MAX_SMEM)
                return VUIB_ERR_SHAPE;
        } else {
            if ((l.mixer != VUIB_LM_MIX_GROUPED && l.mixer != VUIB_LM_MIX_DELTA) || (l.mlp != VUIB_LM_MLP_NONE && l.mlp != VUIB_LM_MLP_RELU2))
                return VUIB_ERR_SHAPE;
            if (l.dim < 1 || l.kv_heads < 1 || l.heads % l.kv_heads) return VUIB_ERR_SHAPE;
            if (l.mixer == VUIB_LM_MIX_GROUPED && (l.rot_dims < 0 || l.rot_dims > l.dim || l.rot_dims % 2 || l.window < 0 ||
                                                   !(l.softcap >= 0.f) || l.dim > GA_MAX_DIM || l.vdim > GA_MAX_DIM))
                return VUIB_ERR_SHAPE;
            if (l.mixer == VUIB_LM_MIX_DELTA && (l.taps < 1 || l.dim > DR_MAX_DIM || l.vdim > DR_MAX_VDIM || l.heads > 65535)) return VUIB_ERR_SHAPE;
        }
    }
    VuibLm* e = new (std::nothrow) VuibLm();
    if (!e) return VUIB_ERR_NULL;
    e->cfg = c;
    e->layer.assign(layers, layers + c.n_layers);
    for (const VuibLmLayer& l : e->layer) {
        e->dims.push_back(layer_dims(c, l));
        e->recurrent = e->recurrent || l.mixer == VUIB_LM_MIX_DELTA;
    }
    e->w.resize(c.n_layers);
    e->maps.resize(c.n_layers);
    e->cache.resize(c.n_layers);
    e->R = c.max_rows > c.max_prefill_rows ? c.max_rows : c.max_prefill_rows;
    e->spin_limit = TC_SPIN_LIMIT;
    e->expand_min = LM_EXPAND_MIN;
    e->few_rows = few_rows_of(e);
    make_layout(e);
    *out = e;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_destroy(VuibLm* e) {
    delete e;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_last_error(VuibLm* e, char* buf, size_t n) {
    if (!e || !buf || n == 0) return VUIB_ERR_NULL;
    strncpy(buf, e->err, n - 1);
    buf[n - 1] = 0;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_layer_dims(VuibLm* e, int32_t layer, VuibLmDims* out) {
    if (!e || !out) return VUIB_ERR_NULL;
    if (layer < 0 || layer >= e->cfg.n_layers) return fail(e, VUIB_ERR_RANGE, "layer %d out of range", layer);
    *out = e->dims[layer];
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_workspace_bytes(VuibLm* e, size_t* bytes) {
    if (!e || !bytes) return VUIB_ERR_NULL;
    *bytes = e->lay.total;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_bind_workspace(VuibLm* e, void* dev, size_t bytes) {
    if (!e || !dev) return VUIB_ERR_NULL;
    if (bytes < e->lay.total || ((uintptr_t)dev & 255))
        return fail(e, VUIB_ERR_WORKSPACE, "workspace needs %zu bytes, 256-byte aligned; got %zu at %p", e->lay.total, bytes, dev);
    e->ws = static_cast<unsigned char*>(dev);
    e->have_ws = true;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_bind_weights(VuibLm* e, const VuibLmHeadWeights* head, const VuibLmLayerWeights* layers) {
    if (!e || !head || !layers) return VUIB_ERR_NULL;
    const VuibLmConfig& c = e->cfg;
    if (!head->embed || !head->final_w || (c.block == VUIB_LM_BLOCK_LN2 && !head->final_b) || !head->head) return fail(e, VUIB_ERR_NULL, "a head weight is NULL");
    for (int i = 0; i < c.n_layers; ++i) {
        const VuibLmLayerWeights& w = layers[i];
        const VuibLmDims& d = e->dims[i];
        const int mixer = e->layer[i].mixer;
        bool have = w.norm1_w && w.w_in && w.w_out && (!e->layer[i].rot_dims || w.trig);
        if (mixer == VUIB_LM_MIX_LATENT)
            have = have && w.norm1_b && (e->layer[i].mlp == VUIB_LM_MLP_NONE || (w.norm2_w && w.norm2_b)) && w.q_norm && w.kv_norm && w.w_q &&
                   w.w_uv && (!d.x_ok || (w.w_xq && w.w_xkv));
        if (mixer == VUIB_LM_MIX_DELTA) have = have && w.conv && w.neg_a && w.dt_bias && w.head_norm;
        if (!have) return fail(e, VUIB_ERR_NULL, "a weight of layer %d is NULL", i);
        e->w[i] = w;
        if (c.dtype == VUIB_LM_BF16) {
            LmMaps& m = e->maps[i];
            bool ok = make_map(&m.w_in, w.w_in, d.n_in, d.k_in, 64) && make_map(&m.w_out, w.w_out, d.n_out, d.k_out, 64);
            if (mixer == VUIB_LM_MIX_LATENT) ok = ok && make_map(&m.w_q, w.w_q, d.n_q, d.k_q, 64);
            if (d.x_ok) ok = ok && make_map(&m.w_xq, w.w_xq, d.n_xq, d.k_q, 64) && make_map(&m.w_xkv, w.w_xkv, d.n_xkv, d.k_kv, 64);
            if (!ok) return fail(e, VUIB_ERR_CUDA, "cuTensorMapEncodeTiled failed for layer %d", i);
        }
    }
    e->head = *head;
    if (c.dtype == VUIB_LM_BF16 && !make_map(&e->map_head, head->head, up(c.vocab, 128), up(c.width, 64), 64))
        return fail(e, VUIB_ERR_CUDA, "cuTensorMapEncodeTiled failed for the head");
    e->have_w = true;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_bind_cache(VuibLm* e, void* const* cache_dev, int32_t* seq_lens_dev) {
    if (!e || !cache_dev || !seq_lens_dev) return VUIB_ERR_NULL;
    for (int i = 0; i < e->cfg.n_layers; ++i) {
        if (!cache_dev[i]) return fail(e, VUIB_ERR_NULL, "cache pointer of layer %d is NULL", i);
        e->cache[i] = cache_dev[i];
    }
    e->seq_lens = seq_lens_dev;
    e->have_cache = true;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_prefill(VuibLm* e, int32_t n_segs, const int32_t* slot, const int32_t* pos, const int32_t* len,
                                   const int64_t* tokens_dev, int32_t n_want, const int32_t* want_rows_dev, float* logits_out_dev,
                                   void* stream) {
    RC(ready(e));
    if (!slot || !pos || !len || !tokens_dev || (n_want > 0 && (!want_rows_dev || !logits_out_dev))) return VUIB_ERR_NULL;
    const VuibLmConfig& c = e->cfg;
    if (n_segs < 1 || n_want < 0) return fail(e, VUIB_ERR_RANGE, "n_segs %d / n_want %d out of range", n_segs, n_want);
    std::vector<int4> segs;
    int rows = 0;
    if (e->recurrent) {
        std::vector<int32_t> slots(slot, slot + n_segs);
        std::sort(slots.begin(), slots.end());
        if (std::adjacent_find(slots.begin(), slots.end()) != slots.end())
            return fail(e, VUIB_ERR_RANGE, "a slot appears twice in a call of a model with recurrent layers");
    }
    for (int i = 0; i < n_segs; ++i) {
        if (slot[i] < 0 || slot[i] >= c.n_slots || pos[i] < 0 || len[i] < 1 || len[i] > c.max_seq || pos[i] > c.max_seq - len[i])
            return fail(e, VUIB_ERR_RANGE, "portion %d: slot %d, positions %d + %d out of range", i, slot[i], pos[i], len[i]);
        if (len[i] > c.max_prefill_rows - rows)
            return fail(e, VUIB_ERR_RANGE, "the portions have more than %d rows", c.max_prefill_rows);
        segs.push_back(make_int4(slot[i], pos[i], len[i], rows));
        rows += len[i];
    }
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    CK(cudaMemcpyAsync(e->ws + e->lay.segs, segs.data(), segs.size() * sizeof(int4), cudaMemcpyHostToDevice, s));
    const bool forms = c.dtype == VUIB_LM_BF16 && rows >= e->expand_min && rows > e->few_rows;
    std::vector<ExpandGroup> groups;
    std::vector<int4> xsegs, tiles;
    if (forms && c.block == VUIB_LM_BLOCK_RMS) {
        for (const int4& g : segs)
            for (int r = (g.z - 1) / GP_TILE * GP_TILE; r >= 0; r -= GP_TILE) {
                tiles.push_back(make_int4(g.w + r, g.z - r < GP_TILE ? g.z - r : GP_TILE, g.x, g.y + r));
                tiles.push_back(make_int4(0, 0, 0, 0));
            }
    } else if (forms && e->lay.x_rows) {
        // sequences are expanded together while their keys fit the scratch (one sequence always does); tiles with the
        // most keys first
        for (const int4& g : segs) {
            const int keys = g.y + g.z;
            if (groups.empty() || groups.back().rows + keys > e->lay.x_rows)
                groups.push_back(ExpandGroup{(int)tiles.size() / 2, 0, (int)xsegs.size(), 0, 0});
            ExpandGroup& q = groups.back();
            for (int r = (g.z - 1) / LP_TILE * LP_TILE; r >= 0; r -= LP_TILE) {
                tiles.push_back(make_int4(g.w + r, g.z - r < LP_TILE ? g.z - r : LP_TILE, g.x, g.y + r));
                tiles.push_back(make_int4(q.rows, 0, 0, 0));
                ++q.n_tiles;
            }
            xsegs.push_back(make_int4(g.x, keys, q.rows, 0));
            ++q.n_segs;
            q.rows += keys;
        }
    }
    if (!xsegs.empty()) CK(cudaMemcpyAsync(e->ws + e->lay.xsegs, xsegs.data(), xsegs.size() * sizeof(int4), cudaMemcpyHostToDevice, s));
    if (!tiles.empty()) CK(cudaMemcpyAsync(e->ws + e->lay.tiles, tiles.data(), tiles.size() * sizeof(int4), cudaMemcpyHostToDevice, s));
    const Pass ps{rows, false, n_segs, (int)tiles.size() / 2, groups.empty() ? nullptr : &groups, false};
    if (c.dtype == VUIB_LM_BF16) return prefill<bf16>(e, ps, tokens_dev, n_want, want_rows_dev, logits_out_dev, s);
    return prefill<float>(e, ps, tokens_dev, n_want, want_rows_dev, logits_out_dev, s);
}

extern "C" int32_t vuib_lm_decode(VuibLm* e, int32_t B, const int32_t* slots_dev, const int32_t* seq_inc_dev,
                                  const int64_t* tokens_dev, float* logits_out_dev, void* stream) {
    RC(ready(e));
    if (!slots_dev || !tokens_dev || !logits_out_dev) return VUIB_ERR_NULL;
    if (B < 1 || B > e->cfg.max_rows) return fail(e, VUIB_ERR_RANGE, "B %d outside [1, %d]", B, e->cfg.max_rows);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (e->cfg.dtype == VUIB_LM_BF16) return decode<bf16>(e, B, slots_dev, seq_inc_dev, tokens_dev, logits_out_dev, s);
    return decode<float>(e, B, slots_dev, seq_inc_dev, tokens_dev, logits_out_dev, s);
}

extern "C" int32_t vuib_lm_set_sampling(VuibLm* e, const VuibSampling* sp, void* stream) {
    if (!e || !sp) return VUIB_ERR_NULL;
    if (!e->have_ws) return fail(e, VUIB_ERR_UNBOUND, "bind the workspace first");
    if (!(sp->temperature > 0.f)) return fail(e, VUIB_ERR_RANGE, "temperature must be > 0");
    if (sp->top_k_cb0 < 0) return fail(e, VUIB_ERR_RANGE, "top_k must be >= 0");
    if (sp->rep_window < 0 || sp->rep_window > REP_HIST_MAX)
        return fail(e, VUIB_ERR_RANGE, "rep_window must be in [0, %d]", REP_HIST_MAX);
    SamplingCtl ctl;
    memset(&ctl, 0, sizeof(ctl));
    ctl.temperature = sp->temperature;
    ctl.top_k_cb0 = sp->top_k_cb0;
    ctl.rep_penalty = sp->rep_penalty;
    ctl.rep_window = sp->rep_window;
    ctl.seed_lo = (uint32_t)(sp->seed & 0xffffffffu);
    ctl.seed_hi = (uint32_t)(sp->seed >> 32);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    CK(cudaMemcpyAsync(e->ws + e->lay.ctl, &ctl, sizeof(ctl), cudaMemcpyHostToDevice, s));
    CK(cudaStreamSynchronize(s));  // the source is a stack object
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_sample(VuibLm* e, int32_t B, const int32_t* slots_dev, float* logits_dev, int64_t* tokens_out_dev,
                                  void* stream) {
    if (!e || !slots_dev || !logits_dev || !tokens_out_dev) return VUIB_ERR_NULL;
    if (!e->have_ws) return fail(e, VUIB_ERR_UNBOUND, "bind the workspace first");
    if (B < 1 || B > e->cfg.max_rows) return fail(e, VUIB_ERR_RANGE, "B %d outside [1, %d]", B, e->cfg.max_rows);
    const LmLayout& L = e->lay;
    const TokenSampleArgs a{logits_dev, e->cfg.vocab, wsp<SamplingCtl>(e, L.ctl), slots_dev, wsp<int32_t>(e, L.draw_ctr),
                            wsp<float>(e, L.rep_counts), wsp<int32_t>(e, L.rep_hist), wsp<int32_t>(e, L.rep_head),
                            wsp<int32_t>(e, L.rep_filled), tokens_out_dev, e->cfg.n_slots, wsp<int32_t>(e, L.flag)};
    return run(e, k_sample_tokens, dim3(B), SAMPLE_THREADS, 0, static_cast<cudaStream_t>(stream), a);
}

extern "C" int32_t vuib_lm_reset_slot(VuibLm* e, int32_t slot, void* stream) {
    if (!e) return VUIB_ERR_NULL;
    if (!e->have_ws) return fail(e, VUIB_ERR_UNBOUND, "bind the workspace first");
    const VuibLmConfig& c = e->cfg;
    if (slot < -1 || slot >= c.n_slots) return fail(e, VUIB_ERR_RANGE, "slot %d out of range", slot);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const LmLayout& L = e->lay;
    const size_t first = slot < 0 ? 0 : slot, n = slot < 0 ? c.n_slots : 1;
    CK(cudaMemsetAsync(e->ws + L.draw_ctr + first * 4, 0, n * 4, s));
    CK(cudaMemsetAsync(e->ws + L.rep_counts + first * c.vocab * 4, 0, n * c.vocab * 4, s));
    CK(cudaMemsetAsync(e->ws + L.rep_hist + first * REP_HIST_MAX * 4, 0, n * REP_HIST_MAX * 4, s));
    CK(cudaMemsetAsync(e->ws + L.rep_head + first * 4, 0, n * 4, s));
    CK(cudaMemsetAsync(e->ws + L.rep_filled + first * 4, 0, n * 4, s));
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_set_taps(VuibLm* e, float* layer_rows_dev) {
    if (!e) return VUIB_ERR_NULL;
    e->taps = layer_rows_dev;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_set_expand_min(VuibLm* e, int32_t rows) {
    if (!e) return VUIB_ERR_NULL;
    if (rows < 0) return fail(e, VUIB_ERR_RANGE, "rows must be >= 0");
    e->expand_min = rows ? rows : LM_EXPAND_MIN;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_set_wait_limit(VuibLm* e, uint32_t polls) {
    if (!e) return VUIB_ERR_NULL;
    if (polls < 16) return fail(e, VUIB_ERR_RANGE, "wait limit %u below 16 polls", polls);
    e->spin_limit = polls;
    return VUIB_OK;
}

extern "C" int32_t vuib_lm_check_device_flag(VuibLm* e, void* stream) {
    if (!e) return VUIB_ERR_NULL;
    if (!e->have_ws) return fail(e, VUIB_ERR_UNBOUND, "bind the workspace first");
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    int32_t flag = 0;
    CK(cudaMemcpyAsync(&flag, e->ws + e->lay.flag, 4, cudaMemcpyDeviceToHost, s));
    CK(cudaStreamSynchronize(s));
    if (flag) {
        CK(cudaMemsetAsync(e->ws + e->lay.flag, 0, 4, s));
        CK(cudaMemsetAsync(e->ws + e->lay.tc_counters, 0, 2 * TC_COUNTERS * 4, s));
        return fail(e, VUIB_ERR_DEVICE_FLAG, "device flag 0x%x (1 = slot outside the cache, 2 = position outside [0, max_seq), 4 = token outside the vocabulary, 16 = a bounded wait inside a kernel ran out)", flag);
    }
    return VUIB_OK;
}

extern "C" int64_t vuib_lm_launch_count(VuibLm* e) { return e ? e->launches : 0; }
