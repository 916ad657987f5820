// Host-side helpers shared by the translation units that launch the decode and token-model kernels:
// programmatic dependent launches, tensor maps, and the launch of the tcgen05 GEMM (tc_gemm.cuh).
#pragma once
#include <cstdlib>
#include <mutex>
#include <unordered_set>

#include "tc_gemm.cuh"

namespace vuib {

constexpr int TC_PARTIAL_TILES = 224;  // most (tile, split) pairs of one GEMM launch
static size_t align_up(size_t v) { return (v + 255) & ~(size_t)255; }


// Launch with the programmatic-stream-serialization attribute (see pdl_wait in
// decode_kernels.cuh) unless VUIB_NO_PDL is set in the environment.
static bool env_off(const char* name) {
    const char* s = getenv(name);
    return s && s[0] && s[0] != '0';
}

static bool pdl_enabled() {
    static int v = -1;
    if (v < 0) {
        const char* s = getenv("VUIB_NO_PDL");
        v = (s && s[0] && s[0] != '0') ? 0 : 1;
    }
    return v == 1;
}

// Every kernel of a frame asks for the same (largest) shared-memory carve-out.  The tensor-core
// GEMM needs ~100-200 KB of shared memory and the small kernels between two GEMMs need almost
// none; left to their own preferences the SMs would re-partition L1/shared memory at every
// switch, which drains them and blocks the overlap of consecutive launches.
static void prefer_max_smem(const void* kern) {
    static std::mutex mu;
    static std::unordered_set<const void*> done;
    std::lock_guard<std::mutex> lock(mu);
    if (done.insert(kern).second)
        cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
}

// `cluster_x` > 1 groups that many consecutive CTAs of the grid's x dimension into a cluster.
template <class... KArgs, class... Args>
static cudaError_t launch_cl(void (*kern)(KArgs...), dim3 grid, int cluster_x, dim3 block, size_t smem, cudaStream_t s,
                             Args... args) {
    prefer_max_smem(reinterpret_cast<const void*>(kern));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (cluster_x > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster_x;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (pdl_enabled()) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}

template <class... KArgs, class... Args>
static cudaError_t launch(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
    return launch_cl(kern, grid, 1, block, smem, s, args...);
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFn encode_tiled_fn() {
    static EncodeTiledFn fn = nullptr;
    static bool tried = false;
    if (!tried) {
        tried = true;
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(p);
    }
    return fn;
}

// 2-D bf16 row-major (rows, cols) tensor, rows `ld` elements apart (cols when 0), boxes of box_rows x 64 columns,
// 128-byte swizzle.
static bool make_map(CUtensorMap* m, const void* ptr, uint64_t rows, uint64_t cols, uint32_t box_rows, uint64_t ld = 0) {
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn) return false;
    cuuint64_t dims[2] = {cols, rows};
    cuuint64_t strides[1] = {(ld ? ld : cols) * 2};
    cuuint32_t box[2] = {TC_KCHUNK, box_rows};
    cuuint32_t estr[2] = {1, 1};
    return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// 2-D bf16 row-major (rows, cols) tensor, dense boxes of box_rows x box_cols, no swizzle.
static bool make_map_plain(CUtensorMap* m, const void* ptr, uint64_t rows, uint64_t cols, uint32_t box_rows,
                           uint32_t box_cols) {
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn || box_rows > 256 || box_cols > 256) return false;
    cuuint64_t dims[2] = {cols, rows};
    cuuint64_t strides[1] = {cols * 2};
    cuuint32_t box[2] = {box_cols, box_rows};
    cuuint32_t estr[2] = {1, 1};
    return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// What one tcgen05 GEMM launch borrows from the engine that issues it.
struct TcCtx {
    float* partial;             // split-K scratch, tc_partial_bytes()
    int32_t* counters;          // 2 x TC_COUNTERS, zero between launches
    int32_t* flag;
    unsigned long long* dbg;    // optional stamps (VUIB_TRACE)
    int* num_sms;               // cached SM count, 0 until the first launch
    unsigned spin_limit;
    long long* launches;
};
constexpr int TC_COUNTERS = 256;

static inline size_t tc_partial_bytes(size_t max_rows) {
    return (size_t)(TC_PARTIAL_TILES + 80) * TC_TILE_N * (max_rows < 256 ? ((max_rows + 15) / 16) * 16 : 256) * 4;
}

// Epilogue staging per activation row: what the functor says, TC_EPI_BYTES_PER_M when it does not.
template <class Epi>
static auto tc_stage_bytes(const Epi& ep, int) -> decltype(ep.stage_bytes_per_row()) { return ep.stage_bytes_per_row(); }
template <class Epi>
static size_t tc_stage_bytes(const Epi&, long) { return TC_EPI_BYTES_PER_M; }

// D = W X^T over all M rows in blocks of <= 256, epilogue ep (see tc_gemm.cuh).
//  units: weight rows (N, multiple of 128) or, for the paired SwiGLU form, hidden units (multiple of 64).
//  x_split_tile / x_split_row: weight tiles from x_split_tile on multiply the M rows that start x_split_row rows
//  further down in X (two inputs of one launch).
template <class Epi>
static cudaError_t tc_gemm_launch(const TcCtx& cx, const CUtensorMap& a0, const CUtensorMap& a1, const bf16* X, int ldx,
                                  int M, int K, int units, int row_off, const Epi& ep, cudaStream_t s,
                                  int x_split_tile = 1 << 30, int x_split_row = 0) {
    const int tiles = Epi::PAIRED ? units / 64 : units / TC_TILE_N;
    const int chunks_total = K / TC_KCHUNK;
    cudaError_t err;
    // Split K over enough CTAs to occupy the SMs (one MMA of this shape takes ~96 ns whatever the
    // batch, so the tensor pipe of ONE SM consumes weights at only ~42 GB/s).  The CTAs of a tile
    // meet on a counter, so the grid must be resident at once: at most two CTAs per SM.
    if (*cx.num_sms == 0) {
        int dev = 0;
        if ((err = cudaGetDevice(&dev)) != cudaSuccess) return err;
        if ((err = cudaDeviceGetAttribute(cx.num_sms, cudaDevAttrMultiProcessorCount, dev)) != cudaSuccess) return err;
    }
    // Row blocks: up to 256 activation rows per CTA; a prefill of more rows is ONE launch whose grid's z
    // dimension walks the blocks (every weight tile is then read by its row blocks back to back and stays in
    // L2), not one launch per block.
    const int Mpad = M <= 256 ? (M + 15) / 16 * 16 : 256;
    const int m_blocks = (M + Mpad - 1) / Mpad;
    int splits = 1;
    for (int d = 2; d <= 16; d *= 2) {
        if (d > chunks_total || tiles * m_blocks * d > *cx.num_sms + *cx.num_sms / 2) break;
        if (Epi::PAIRED && d == 2) continue;
        splits = d;
    }
    const int max_smem = 202 * 1024;
    {   // a function attribute belongs to one device's copy of the kernel: set it once per device
        static std::mutex mu;
        static bool attr_set[64];
        int dev = 0;
        if ((err = cudaGetDevice(&dev)) != cudaSuccess) return err;
        std::lock_guard<std::mutex> lock(mu);
        if (dev < 0 || dev >= 64 || !attr_set[dev]) {
            if ((err = cudaFuncSetAttribute(k_gemm_tc<Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem)) != cudaSuccess)
                return err;
            if (dev >= 0 && dev < 64) attr_set[dev] = true;
        }
    }
    CUtensorMap mx;
    if (!make_map(&mx, X, (uint64_t)M + x_split_row, K, Mpad, ldx)) return cudaErrorInvalidValue;
    TcArgs ta;
    ta.N = units;
    ta.row_off = row_off;
    ta.M = M;
    ta.Mpad = Mpad;
    ta.chunks = chunks_total;
    ta.splits = splits;
    ta.tiles = tiles;
    ta.partial = cx.partial;
    ta.counters = cx.counters;
    ta.flag = cx.flag;
    ta.dbg = cx.dbg;
    ta.spin_limit = cx.spin_limit;
    ta.x_split_tile = x_split_tile;
    ta.x_split_row = x_split_row;
    const int min_chunks = chunks_total / splits;  // the shortest split
    const size_t stage_bytes = TC_TILE_N * TC_KCHUNK * 2 + ((Mpad * TC_KCHUNK * 2 + 1023) & ~1023);
    const size_t epi_bytes = Epi::STAGED ? (size_t)Mpad * tc_stage_bytes(ep, 0) : 0;
    // two CTAs per SM when split (all CTAs of the grid must be resident), the whole SM otherwise
    const size_t budget = (splits > 1 ? 100 : 200) * 1024;
    int stages = epi_bytes + stage_bytes <= budget ? (int)((budget - epi_bytes) / stage_bytes) : 1;
    if (stages > TC_MAX_STAGES) stages = TC_MAX_STAGES;
    if (stages > min_chunks) stages = min_chunks;
    ta.stages = stages;
    const size_t smem = (size_t)stages * stage_bytes + epi_bytes + 1024;
    ++*cx.launches;
    return launch(k_gemm_tc<Epi>, dim3(splits, tiles, m_blocks), TC_THREADS, smem, s, a0, a1, mx, ta, ep);
}


}  // namespace vuib
