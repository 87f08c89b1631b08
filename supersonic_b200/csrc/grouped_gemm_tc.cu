// Grouped matrix products for sm_100a (tcgen05): for every expert e, C[rows of e] = A[rows of e] W_e^T, bfloat16 in, float32
// accumulators in tensor memory.  The rows of A are sorted by expert; a device-side tile list names the runs of up to NT
// rows of one expert.
//
// The weights take the M side of the product: a work item is 128 rows of an expert's W (128 columns of C) times the rows of
// one tile, which take the N side.  How many rows a tile has varies from one to NT, and so does the N of its tcgen05.mma (a
// multiple of 16): a group of 180 rows costs 192 columns of tensor work, a decode step's group of two rows costs 16 while
// its weights stream through once.  Operands arrive through TMA (128-byte swizzle) into a ring of stages; the rows of A
// come in boxes of BOX rows, as many as the tile needs (rows behind a tile's end belong to the next expert and are never
// stored).  Accumulators of consecutive items alternate between two regions of tensor memory, so that the epilogue of one
// overlaps the MMAs of the next.
//
// Epilogues: store as bfloat16 or float32, through an activation, or the gated unit: W_e is [gate rows; up rows], a warp's
// 32 accumulator lanes are 16 gate rows and the 16 up rows of the same columns, and the two meet by a shuffle.  Rows of C
// may be scattered through an index.
//
// The same kernel takes one matrix per head (C[t, h] = W_h A[t, h] for all tokens t): the heads' columns sit side by side in a
// row of A and of C, tiles are cut from the tokens, and the epilogue may multiply by the sigmoid of a gate's element.
//
// Every wait on an mbarrier is bounded: when one runs out, the block records a code in the caller's error word, lets its
// copies land, frees its tensor memory and returns.
#include "common.cuh"
#include "tc_helpers.cuh"

typedef __nv_bfloat16 bf16;

constexpr int GT_THREADS = 192;           // warp 0: TMA, warp 1: MMA + tensor memory, warps 2-5: epilogue
constexpr int GT_BM = 128;
constexpr int GT_TILE_LD = 36;            // padded row of an epilogue warp's 32 x 32 tile in shared memory
enum { GT_STORE = 0, GT_GATED = 1, GT_ACT = 2, GT_HEADS = 3 };

struct GtArgs {
    const int* offsets; const int* tile_expert; const int* tile_row0; const int* meta;
    void* C; int ldc; const int* c_index;
    int N, K, w_rows, n_cols;             // columns of C, inner size, rows of one expert's W, column items a tile has
    int kind; float limit;                // activation or inner step of the gated unit
    int* error_word;
    int vec;                              // rows of C are whole 16-byte pieces
    int a_batch, c_batch, n_rows, n_heads; const bf16* gate; int ldg;   // GT_HEADS: columns between heads of A and C, tokens, gates
};

template <int MODE>
struct GtItem {
    int e, r0, rows, col;
    __device__ __forceinline__ static GtItem at(const GtArgs& g, int item, int total, int nt) {
        GtItem x;
        x.e = x.r0 = x.rows = x.col = 0;
        if (MODE == GT_HEADS) {                           // the heads of a tile of tokens in a row, so that the tokens' rows stay near
            if (item < total) {
                const int rest = item / g.n_cols;
                x.col = item - rest * g.n_cols;
                x.e = rest % g.n_heads;
                x.r0 = rest / g.n_heads * nt;
                x.rows = min(g.n_rows - x.r0, nt);
            }
        } else if (item < total) {
            const int tile = item / g.n_cols;
            x.col = item - tile * g.n_cols;
            x.e = g.tile_expert[tile];
            x.r0 = g.tile_row0[tile];
            x.rows = min(g.offsets[x.e + 1] - x.r0, nt);
        }
        return x;
    }
};

__device__ __forceinline__ void gt_arrive(uint32_t bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
// V neighbouring values of a row of C: one 16-byte piece, or (columns or rows that are not whole pieces) the first n singly
template <int V, bool F32>
__device__ __forceinline__ void gt_put(void* C, size_t at, const float (&v)[V], int n, bool vec) {
    if (vec) {
        if (F32) {
            *reinterpret_cast<float4*>(reinterpret_cast<float*>(C) + at) = make_float4(v[0], v[1], v[2], v[3]);
        } else {
            uint32_t p[V / 2];
#pragma unroll
            for (int k = 0; k < V; k += 2) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(v[k], v[k + 1]);
                p[k / 2] = *reinterpret_cast<const uint32_t*>(&b);
            }
            *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(C) + at) = make_uint4(p[0], p[1], p[V / 2 - 2], p[V / 2 - 1]);
        }
        return;
    }
#pragma unroll
    for (int k = 0; k < V; ++k)
        if (k < n) {
            if (F32) reinterpret_cast<float*>(C)[at + k] = v[k];
            else reinterpret_cast<bf16*>(C)[at + k] = __float2bfloat16_rn(v[k]);
        }
}

template <int NT, int BOX, int STAGES, int MODE, bool F32>
__global__ void __launch_bounds__(GT_THREADS, 1)
grouped_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_a, const GtArgs g) {
    constexpr uint32_t W_BYTES = GT_BM * TC_BK * 2, A_BYTES = NT * TC_BK * 2, STAGE_BYTES = W_BYTES + A_BYTES;
    constexpr int N_ACC = 2, COLS = MODE == GT_GATED ? 64 : 128, CW = COLS / 4, V = F32 ? 4 : 8, UNITS = CW / V;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    float* tiles = (float*)(smem + STAGES * STAGE_BYTES);           // [4 epilogue warps][32][GT_TILE_LD]
    uint64_t* bars = (uint64_t*)(tiles + 4 * 32 * GT_TILE_LD);
    uint32_t* tmem_slot = (uint32_t*)(bars + 2 * STAGES + 2 * N_ACC);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);     // [0]: a role gave up; [1]: stays zero
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int k_blocks = (g.K + TC_BK - 1) / TC_BK;
    const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
    const uint32_t acc_full0 = smem_u32(bars + 2 * STAGES), acc_empty0 = smem_u32(bars + 2 * STAGES + N_ACC);

    ssb_pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(full0 + 8 * s, 1); mbar_init(empty0 + 8 * s, 1); }
        for (int i = 0; i < N_ACC; ++i) { mbar_init(acc_full0 + 8 * i, 1); mbar_init(acc_empty0 + 8 * i, 4); }
        abort_flag[0] = 0;
        abort_flag[1] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(N_ACC * NT) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    ssb_pdl_wait();                                             // the tile list and the rows of A are there
    const int total = MODE == GT_HEADS ? (g.n_rows + NT - 1) / NT * g.n_heads * g.n_cols : g.meta[0] * g.n_cols;

    if (warp == 0) {
        if (lane == 0) {
            int c = 0;
            for (int item = blockIdx.x; item < total && !*abort_flag; item += gridDim.x) {
                const GtItem<MODE> it = GtItem<MODE>::at(g, item, total, NT);
                const int boxes = (it.rows + BOX - 1) / BOX;
                const uint32_t bytes = W_BYTES + boxes * BOX * TC_BK * 2;
                const int w0 = it.e * g.w_rows + it.col * COLS, x0 = MODE == GT_HEADS ? it.e * g.a_batch : 0;
                for (int kb = 0; kb < k_blocks; ++kb, ++c) {
                    const int s = c % STAGES;
                    const uint32_t phase = (c / STAGES) & 1;
                    if (!mbar_wait(empty0 + 8 * s, phase ^ 1, abort_flag)) {
                        *abort_flag = 1; atomicCAS(g.error_word, 0, TC_ERR_PRODUCER); break;
                    }
                    const uint32_t w_dst = smem_u32(smem + s * STAGE_BYTES), a_dst = w_dst + W_BYTES;
                    mbar_expect_tx(full0 + 8 * s, bytes);
                    if (MODE == GT_GATED) {
#pragma unroll
                        for (int q = 0; q < 4; ++q) {           // 16 gate rows and their 16 up rows for every warp of the epilogue
                            tma_load_2d(w_dst + q * 4096, &map_w, full0 + 8 * s, kb * TC_BK, w0 + q * 16);
                            tma_load_2d(w_dst + q * 4096 + 2048, &map_w, full0 + 8 * s, kb * TC_BK, w0 + g.N + q * 16);
                        }
                    } else {
                        tma_load_2d(w_dst, &map_w, full0 + 8 * s, kb * TC_BK, w0);
                    }
                    for (int b = 0; b < boxes; ++b)
                        tma_load_2d(a_dst + b * BOX * TC_BK * 2, &map_a, full0 + 8 * s, x0 + kb * TC_BK, it.r0 + b * BOX);
                }
            }
            if (*abort_flag)                                    // let copies that were issued but never consumed land
                for (int i = max(0, c - STAGES); i < c; ++i)
                    mbar_wait(full0 + 8 * (i % STAGES), (i / STAGES) & 1, abort_flag + 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = true;
            int c = 0, i = 0;
            GtItem<MODE> next = GtItem<MODE>::at(g, blockIdx.x, total, NT);
            for (int item = blockIdx.x; item < total && ok; item += gridDim.x, ++i) {
                const int n = (next.rows + 15) & ~15;
                next = GtItem<MODE>::at(g, item + gridDim.x, total, NT);
                // instruction descriptor: D float32, A and B bfloat16, both K-major, N the tile's rows, M 128
                const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(GT_BM >> 4) << 24);
                const int buf = i % N_ACC;
                const uint32_t use = (uint32_t)(i / N_ACC) & 1;
                if (!mbar_wait(acc_empty0 + 8 * buf, use ^ 1, abort_flag)) {
                    *abort_flag = 1; atomicCAS(g.error_word, 0, TC_ERR_MMA); ok = false; break;
                }
                tc_fence_after();
                const uint32_t acc = tmem + buf * NT;
                for (int kb = 0; kb < k_blocks && ok; ++kb, ++c) {
                    const int s = c % STAGES;
                    const uint32_t phase = (c / STAGES) & 1;
                    if (!mbar_wait(full0 + 8 * s, phase, abort_flag)) {
                        *abort_flag = 1; atomicCAS(g.error_word, 0, TC_ERR_MMA); ok = false; break;
                    }
                    tc_fence_after();
                    const uint32_t w_addr = smem_u32(smem + s * STAGE_BYTES);
                    static_assert(TC_BK == 64, "four k-steps a k-block");
                    tc_mma_x4(acc, smem_desc(w_addr), smem_desc(w_addr + W_BYTES), idesc, kb > 0 ? 1u : 0u);
                    tc_commit(empty0 + 8 * s);
                }
                if (ok) tc_commit(acc_full0 + 8 * buf);
            }
        }
    } else {
        const int quarter = warp & 3;
        int i = 0;
        for (int item = blockIdx.x; item < total; item += gridDim.x, ++i) {
            const GtItem<MODE> it = GtItem<MODE>::at(g, item, total, NT);
            const int buf = i % N_ACC;
            const uint32_t use = (uint32_t)(i / N_ACC) & 1;
            bool ok = mbar_wait(acc_full0 + 8 * buf, use, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) {
                if (lane == 0) { *abort_flag = 1; atomicCAS(g.error_word, 0, TC_ERR_EPILOGUE); }
                break;
            }
            tc_fence_after();
            const uint32_t acc = tmem + buf * NT + ((uint32_t)(quarter * 32) << 16);
            float* tile = tiles + quarter * 32 * GT_TILE_LD;
            const int n_warp = it.col * COLS + quarter * CW;                 // the warp's first column of C
            for (int c = 0; c < it.rows; c += 32) {
                uint32_t r[32];
                tc_ld32(acc + c, r);
                const int mine = c + lane < it.rows ? it.r0 + c + lane : it.r0;
                const int row = g.c_index ? g.c_index[mine] : mine;          // lane j: where row c + j of the tile goes
                const int here = min(32, it.rows - c);
                // a lane holds one column of 32 rows: through shared memory to whole 16-byte pieces of a row
                if (MODE == GT_GATED) {
                    const bool up = lane >= 16;
#pragma unroll
                    for (int j = 0; j < 32; j += 2) {
                        // lanes 0-15 finish row j, lanes 16-31 row j + 1
                        const float own = __uint_as_float(up ? r[j + 1] : r[j]), give = __uint_as_float(up ? r[j] : r[j + 1]);
                        const float got = __shfl_xor_sync(0xffffffffu, give, 16);
                        tile[(j + (up ? 1 : 0)) * GT_TILE_LD + (lane & 15)] = ssb_gate_fast(up ? got : own, up ? own : got, g.kind, g.limit);
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        const float v = __uint_as_float(r[j]);
                        tile[j * GT_TILE_LD + lane] = MODE == GT_ACT ? ssb_activate(v, g.kind) : v;
                    }
                }
                __syncwarp();
#pragma unroll
                for (int i = 0; i < UNITS; ++i) {
                    const int u = i * 32 + lane, j = u / UNITS, at_n = (u % UNITS) * V, n = n_warp + at_n;
                    const int at = __shfl_sync(0xffffffffu, row, j);
                    if (j < here && n < g.N) {
                        float v[V];
#pragma unroll
                        for (int k = 0; k < V; k += 4) {
                            const float4 q = *reinterpret_cast<const float4*>(tile + j * GT_TILE_LD + at_n + k);
                            v[k] = q.x; v[k + 1] = q.y; v[k + 2] = q.z; v[k + 3] = q.w;
                        }
                        if (MODE == GT_HEADS && g.gate != nullptr) {
                            const bf16* z = g.gate + (size_t)at * g.ldg + it.e * g.N + n;
#pragma unroll
                            for (int k = 0; k < V; ++k)
                                if (n + k < g.N) v[k] = __fdividef(v[k], 1.0f + __expf(-__bfloat162float(z[k])));
                        }
                        gt_put<V, F32>(g.C, (size_t)at * g.ldc + (MODE == GT_HEADS ? it.e * g.c_batch : 0) + n, v, g.N - n, g.vec);
                    }
                }
                __syncwarp();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) gt_arrive(acc_empty0 + 8 * buf);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(N_ACC * NT) : "memory");
    }
}

static int gt_whole(const void* C, int ldc, int c_batch, int N, int out_dtype) {
    const int v = out_dtype == SSB_F32 ? 4 : 8;
    return N % v == 0 && ldc % v == 0 && c_batch % v == 0 && ((uintptr_t)C & 15) == 0;
}

static int gt_sms() {
    static int n_sms = 0;
    if (!n_sms) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess ||
            cudaDeviceGetAttribute(&n_sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n_sms <= 0)
            n_sms = 148;
    }
    return n_sms;
}

template <int NT, int BOX, int STAGES, int MODE, bool F32>
static int gt_launch(const CUtensorMap& mw, const CUtensorMap& ma, const GtArgs& g, long long max_items, int pdl, cudaStream_t stream) {
    constexpr size_t smem = STAGES * (GT_BM + NT) * TC_BK * 2 + 4 * 32 * GT_TILE_LD * 4 + (2 * STAGES + 4) * 8 + 16 + 1024;
    auto kern = grouped_gemm_tc_kernel<NT, BOX, STAGES, MODE, F32>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const int blocks = max_items < gt_sms() ? (int)max_items : gt_sms();
    const int rc = ssb_launch(kern, dim3(blocks), dim3(GT_THREADS), smem, stream, pdl != 0, mw, ma, g);
    return rc ? rc : ssb_launch_status();
}

// One matrix per head: C[t, h * c_batch + n] = sum_k W[h, n, k] A[t, h * a_batch + k], with a gate (bfloat16 [M, n_heads x N])
// times sigmoid(gate[t, h * N + n]).  A's rows hold a_cols columns.  What a head's last k-block reads behind its own columns
// meets the zeros behind W's.
SSB_API int ssb_head_gemm_tc(const void* A, int lda, int a_cols, int a_batch, const void* W, void* C, int ldc, int c_batch,
                             int out_dtype, int n_heads, int M, int N, int K, const void* gate, int ldg, int* error_word, int pdl,
                             cudaStream_t stream) {
    if (M <= 0 || N <= 0 || n_heads <= 0) return 0;
    if (K <= 0 || K % 8 || lda % 8 || a_batch % 8 || a_batch < 0 || (long long)(n_heads - 1) * a_batch + K > a_cols || !error_word ||
        (long long)n_heads * N > 0x7fffff00ll)
        return SSB_ERR_BAD_SIZE;
    if (((uintptr_t)A | (uintptr_t)W) & 15) return SSB_ERR_BAD_SIZE;
    GtArgs g{nullptr, nullptr, nullptr, nullptr, C, ldc, nullptr, N, K, N, (N + 127) / 128, 0, 0.f, error_word, gt_whole(C, ldc, c_batch, N, out_dtype),
             a_batch, c_batch, M, n_heads, (const bf16*)gate, ldg};
    const long long items = (long long)((M + 127) / 128) * n_heads * g.n_cols;
    if (items > 0x7fff0000ll) return SSB_ERR_BAD_SIZE;
    CUtensorMap mw, ma;
    int rc = make_map(&mw, W, n_heads * N, K, K, GT_BM);
    if (rc) return rc;
    rc = make_map(&ma, A, M, a_cols, lda, 64);
    if (rc) return rc;
    if (out_dtype == SSB_F32) return gt_launch<128, 64, 6, GT_HEADS, true>(mw, ma, g, items, pdl, stream);
    if (out_dtype == SSB_BF16) return gt_launch<128, 64, 6, GT_HEADS, false>(mw, ma, g, items, pdl, stream);
    return SSB_ERR_BAD_DTYPE;
}

// A: bfloat16 [n_rows, K] sorted by expert; W: bfloat16 [n_experts, w_rows, K]; tile list of runs of up to tile_rows (64,
// 128 or 256) rows.  mode 0: C = A W_e^T (N = w_rows columns); 1: w_rows = 2 N, gated unit of kind `kind` with clamp
// `limit`, C bfloat16; 2: activation `kind` on the sums, C bfloat16.
SSB_API int ssb_grouped_gemm_tc(const void* A, int lda, const void* W, int n_experts, int w_rows, void* C, int ldc,
                                const int* c_index, int out_dtype, const int* offsets, const int* tile_expert,
                                const int* tile_row0, const int* meta, int max_tiles, int tile_rows, int n_rows, int N, int K,
                                int mode, int kind, float limit, int* error_word, int pdl, cudaStream_t stream) {
    if (max_tiles <= 0 || N <= 0 || n_rows <= 0) return 0;
    if (K <= 0 || K % 8 || lda % 8 || n_experts <= 0 || !error_word || mode < 0 || mode > 2) return SSB_ERR_BAD_SIZE;
    if (w_rows != (mode == GT_GATED ? 2 * N : N) || (long long)n_experts * w_rows > 0x7fffff00ll) return SSB_ERR_BAD_SIZE;
    if (((uintptr_t)A | (uintptr_t)W) & 15) return SSB_ERR_BAD_SIZE;
    if (mode != GT_STORE && out_dtype != SSB_BF16) return SSB_ERR_BAD_DTYPE;
    if (kind < 0 || kind > (mode == GT_ACT ? (int)SSB_ACT_SILU : (int)SSB_GATE_LAST)) return SSB_ERR_BAD_SIZE;
    const int cols = mode == GT_GATED ? 64 : 128;
    GtArgs g{offsets, tile_expert, tile_row0, meta, C, ldc, c_index, N, K, w_rows, (N + cols - 1) / cols, kind, limit, error_word,
             gt_whole(C, ldc, 0, N, out_dtype), 0, 0, 0, 0, nullptr, 0};
    const long long items = (long long)max_tiles * g.n_cols;
    if (items > 0x7fff0000ll) return SSB_ERR_BAD_SIZE;
    CUtensorMap mw, ma;
    int rc = make_map(&mw, W, n_experts * w_rows, K, K, mode == GT_GATED ? 16 : GT_BM);
    if (rc) return rc;
    rc = make_map(&ma, A, n_rows, K, lda, tile_rows == 64 ? 16 : 64);
    if (rc) return rc;
#define SSB_GT(NT, BOX, ST)                                                                                     \
    do {                                                                                                        \
        if (mode == GT_GATED) return gt_launch<NT, BOX, ST, GT_GATED, false>(mw, ma, g, items, pdl, stream);    \
        if (mode == GT_ACT) return gt_launch<NT, BOX, ST, GT_ACT, false>(mw, ma, g, items, pdl, stream);        \
        if (out_dtype == SSB_F32) return gt_launch<NT, BOX, ST, GT_STORE, true>(mw, ma, g, items, pdl, stream); \
        if (out_dtype == SSB_BF16) return gt_launch<NT, BOX, ST, GT_STORE, false>(mw, ma, g, items, pdl, stream); \
        return SSB_ERR_BAD_DTYPE;                                                                               \
    } while (0)
    if (tile_rows == 64) SSB_GT(64, 16, 8);
    if (tile_rows == 128) SSB_GT(128, 64, 6);
    if (tile_rows == 256) SSB_GT(256, 64, 4);
#undef SSB_GT
    return SSB_ERR_BAD_SIZE;
}
