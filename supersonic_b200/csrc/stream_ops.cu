// Several residual streams side by side (hyper-connections).  A token has streams x_1 .. x_S of float32 rows.  A
// sublayer reads one mix of them and its result is written back into all of them, which are mixed with one another
// at the same time:
//     u = sum_s in[s] x_s,      y = sublayer(norm(u)),      x_t <- sum_s mix[s, t] x_s + out[t] y      (mix is [from, to])
//
// Between two sublayers the write of the first and the read of the second are one pass over the streams
// (stream_cross_kernel): read the old streams and the branch y, make the new streams, store them, take the next mix u
// of them, its RMS norm and, in steps of one token a sequence, the short convolution behind the norm.  The branch is
// zeroed behind the read, so that the next sublayer's products can add into it.
//
// Everything is float32 except the normed row that the sublayer reads.
#include "common.cuh"
#include <math.h>

typedef __nv_bfloat16 bf16;

constexpr int SX_MAX_STREAMS = 16;
constexpr int SX_MAX_TAPS = 16;

struct SxArgs {
    const float* src;            // [n_src][tokens][width]: the streams, or (n_src = 1) the one row that all of them equal
    int n_src;
    long long plane;             // elements of a plane of src and dst
    float* branch;               // [tokens][width] y, or null: nothing is written back
    int clear;                   // zero the branch behind the read
    const float* mix;            // [S][S], with a branch
    const float* out_w;          // [S]
    float* dst;                  // [S][tokens][width], or null: the new streams are not stored (may be src)
    const float* in_w;           // [S], or null: the sum of the streams
    const float* norm_w;         // [width], or null: u itself goes out (float32)
    float eps;
    void* out;                   // [tokens][width]
    const float* conv_w;         // [taps][width], or null: no convolution behind the norm
    float* tail;                 // [slots][taps - 1][width] the last taps - 1 normed rows, oldest first
    const int* slot;             // [tokens]
    int taps, width, streams;
};

// The convolution behind the norm, for one column of a token that is alone in its sequence's step.
__device__ __forceinline__ float sx_convolve(const SxArgs& a, int slot, int c, float n) {
    const int back = a.taps - 1;
    const float* w = a.conv_w + c;
    float acc = 0.f;
    if (slot >= 0 && back > 0) {                           // the kept rows move down by one place
        float* keep = a.tail + (size_t)slot * back * a.width + c;
        for (int j = 0; j < back; ++j) {
            const float v = keep[(size_t)j * a.width];
            acc = fmaf(w[(size_t)j * a.width], v, acc);
            if (j > 0) keep[(size_t)(j - 1) * a.width] = v;
        }
        keep[(size_t)(back - 1) * a.width] = n;
    }
    return fmaf(w[(size_t)back * a.width], n, acc);
}

__device__ __forceinline__ float sx_block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
    for (int w = 0; w < (int)blockDim.x / 32; ++w) total += red[w];
    return total;
}

__device__ __forceinline__ void sx_store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void sx_store4(bf16* p, const float* v) {
    const __nv_bfloat162 x = __floats2bfloat162_rn(v[0], v[1]), y = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&x);
    u.y = *reinterpret_cast<const uint32_t*>(&y);
    *reinterpret_cast<uint2*>(p) = u;
}

// Rows of whole float4s that a block's registers hold: everything is loaded before anything is stored (a loop that
// zeroes a piece of the branch between its loads takes ten times as long: 211 against 20 us for 2,048 rows of 2,048
// and two streams).  S: the number of streams; N: float4s a thread owns of a row.
// TAPS > 0: with a convolution of that many taps behind the norm, whose weights and kept rows are requested with the rest.
template <typename T, int S, int N, int NT, int TAPS>
__global__ void __launch_bounds__(NT)
stream_cross_vec_kernel(const SxArgs a) {
    constexpr int BACK = TAPS > 0 ? TAPS - 1 : 0;
    __shared__ float red[32];
    const int tid = threadIdx.x, W = a.width, n4 = W / 4;
    const bool writes = a.branch != nullptr;
    ssb_pdl_launch_dependents();
    // coefficients and the norm's weights: no kernel of a step writes them
    float mix[S * S], out_w[S], in_w[S];
#pragma unroll
    for (int i = 0; i < S * S; ++i) mix[i] = writes ? a.mix[i] : 0.f;
#pragma unroll
    for (int i = 0; i < S; ++i) {
        out_w[i] = writes ? a.out_w[i] : 0.f;
        in_w[i] = a.in_w != nullptr ? a.in_w[i] : 1.0f;
    }
    float4 cw[TAPS > 0 ? TAPS : 1][N], kept[BACK > 0 ? BACK : 1][N];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int c = tid + n * NT;
            if (c < n4) cw[j][n] = *reinterpret_cast<const float4*>(a.conv_w + (size_t)j * W + 4 * c);
        }
    ssb_pdl_wait();
    const size_t row = (size_t)blockIdx.x * W;
    const int slot = TAPS > 0 ? a.slot[blockIdx.x] : -1;
    float* keep = BACK > 0 && slot >= 0 ? a.tail + (size_t)slot * BACK * W : nullptr;
#pragma unroll
    for (int j = 0; j < BACK; ++j)
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int c = tid + n * NT;
            kept[j][n] = keep != nullptr && c < n4 ? *reinterpret_cast<const float4*>(keep + (size_t)j * W + 4 * c)
                                                   : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    float x[S][N][4], y[N][4];
#pragma unroll
    for (int n = 0; n < N; ++n) {
        const int c = tid + n * NT;
        const size_t at = row + 4 * (size_t)c;
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if (s > 0 && a.n_src == 1) {
#pragma unroll
                for (int k = 0; k < 4; ++k) x[s][n][k] = x[0][n][k];
                continue;
            }
            const float4 v = c < n4 ? *reinterpret_cast<const float4*>(a.src + s * a.plane + at) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[s][n][0] = v.x; x[s][n][1] = v.y; x[s][n][2] = v.z; x[s][n][3] = v.w;
        }
        const float4 v = writes && c < n4 ? *reinterpret_cast<const float4*>(a.branch + at) : make_float4(0.f, 0.f, 0.f, 0.f);
        y[n][0] = v.x; y[n][1] = v.y; y[n][2] = v.z; y[n][3] = v.w;
    }
    float sq = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            float u = 0.f;
            if (writes) {
                float v[S];
#pragma unroll
                for (int to = 0; to < S; ++to) {
                    v[to] = out_w[to] * y[n][k];
#pragma unroll
                    for (int s = 0; s < S; ++s) v[to] = fmaf(mix[s * S + to], x[s][n][k], v[to]);
                    u = fmaf(in_w[to], v[to], u);
                }
#pragma unroll
                for (int to = 0; to < S; ++to) x[to][n][k] = v[to];
            } else {
#pragma unroll
                for (int s = 0; s < S; ++s) u = fmaf(in_w[s], x[s][n][k], u);
            }
            y[n][k] = u;
            sq = fmaf(u, u, sq);
        }
#pragma unroll
    for (int n = 0; n < N; ++n) {
        const int c = tid + n * NT;
        const size_t at = row + 4 * (size_t)c;
        if (c >= n4) continue;
        if (a.dst != nullptr)
#pragma unroll
            for (int s = 0; s < S; ++s) sx_store4(a.dst + s * a.plane + at, x[s][n]);
        if (writes && a.clear) *reinterpret_cast<float4*>(a.branch + at) = make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.norm_w == nullptr) sx_store4(reinterpret_cast<float*>(a.out) + at, y[n]);
    }
    if (a.norm_w == nullptr) return;
    const float inv = 1.0f / sqrtf(sx_block_sum(sq, red) / (float)W + a.eps);
#pragma unroll
    for (int n = 0; n < N; ++n) {
        const int c = tid + n * NT;
        if (c >= n4) continue;
        const float4 w = *reinterpret_cast<const float4*>(a.norm_w + 4 * c);
        float v[4] = {y[n][0] * inv * w.x, y[n][1] * inv * w.y, y[n][2] * inv * w.z, y[n][3] * inv * w.w};
        if (TAPS > 0) {
            const float4 now = make_float4(v[0], v[1], v[2], v[3]);
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                const float4 r = j < BACK ? kept[j < BACK ? j : 0][n] : now;
                acc[0] = fmaf(cw[j][n].x, r.x, acc[0]); acc[1] = fmaf(cw[j][n].y, r.y, acc[1]);
                acc[2] = fmaf(cw[j][n].z, r.z, acc[2]); acc[3] = fmaf(cw[j][n].w, r.w, acc[3]);
            }
            if (keep != nullptr)
#pragma unroll
                for (int j = 0; j < BACK; ++j)             // the kept rows move down by one place
                    *reinterpret_cast<float4*>(keep + (size_t)j * W + 4 * c) = j + 1 < BACK ? kept[j + 1 < BACK ? j + 1 : 0][n] : now;
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = acc[k];
        }
        sx_store4(reinterpret_cast<T*>(a.out) + row + 4 * c, v);
    }
}

// Any width and number of streams (SM: an upper bound of it, the loops over the streams are unrolled).  u's row waits in
// shared memory for its sum of squares, which is taken in a fixed order.
template <typename T, int SM>
__global__ void stream_cross_kernel(const SxArgs a) {
    extern __shared__ float sx_row[];
    __shared__ float red[32];
    __shared__ float c_mix[SM * SM], c_out[SM], c_in[SM];
    const int tid = threadIdx.x, nt = blockDim.x, S = a.streams, W = a.width;
    const bool writes = a.branch != nullptr;
    ssb_pdl_launch_dependents();
    if (writes) {
        for (int i = tid; i < S * S; i += nt) c_mix[(i / S) * SM + i % S] = a.mix[i];
        for (int i = tid; i < S; i += nt) c_out[i] = a.out_w[i];
    }
    for (int i = tid; i < S; i += nt) c_in[i] = a.in_w != nullptr ? a.in_w[i] : 1.0f;
    ssb_pdl_wait();
    __syncthreads();
    const size_t t = blockIdx.x;
    const float* src = a.src + t * W;
    float* br = writes ? a.branch + t * W : nullptr;
    float sq = 0.f;
    for (int c = tid; c < W; c += nt) {
        float x[SM];
#pragma unroll
        for (int s = 0; s < SM; ++s) x[s] = s < S ? src[(a.n_src > 1 ? (size_t)s * a.plane : 0) + c] : 0.f;
        float u = 0.f;
        if (writes) {
            const float y = br[c];
#pragma unroll
            for (int to = 0; to < SM; ++to)
                if (to < S) {
                    float v = c_out[to] * y;
#pragma unroll
                    for (int s = 0; s < SM; ++s)
                        if (s < S) v = fmaf(c_mix[s * SM + to], x[s], v);
                    if (a.dst != nullptr) a.dst[(size_t)to * a.plane + t * W + c] = v;
                    u = fmaf(c_in[to], v, u);
                }
        } else {
#pragma unroll
            for (int s = 0; s < SM; ++s)
                if (s < S) u = fmaf(c_in[s], x[s], u);
        }
        if (a.norm_w == nullptr) reinterpret_cast<float*>(a.out)[t * W + c] = u;
        else sx_row[c] = u;
        sq = fmaf(u, u, sq);
    }
    if (writes && a.clear)
        for (int c = tid; c < W; c += nt) br[c] = 0.f;
    if (a.norm_w == nullptr) return;
    const float inv = 1.0f / sqrtf(sx_block_sum(sq, red) / (float)W + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + t * W;
    const int slot = a.conv_w != nullptr ? a.slot[t] : -1;
    for (int c = tid; c < W; c += nt) {
        const float n = sx_row[c] * inv * a.norm_w[c];
        out[c] = ssb_from_float<T>(a.conv_w != nullptr ? sx_convolve(a, slot, c, n) : n);
    }
}

constexpr int SX_VEC_TAPS = 4;                             // taps the kernel above holds in registers

template <typename T, int S, int TAPS>
static int launch_stream_vec(const SxArgs& a, int n_tokens, bool pdl, cudaStream_t stream) {
    const int n4 = a.width / 4;
#define SSB_SXV(N, NT) return ssb_launch(stream_cross_vec_kernel<T, S, N, NT, TAPS>, dim3(n_tokens), dim3(NT), 0, stream, pdl, a)
    if (n4 <= 128) SSB_SXV(1, 128);
    if (n4 <= 256) SSB_SXV(1, 256);
    if (n4 <= 512) SSB_SXV(1, 512);
    if (n4 <= 1024) SSB_SXV(2, 512);
    if constexpr (TAPS == 0) { SSB_SXV(4, 512); }
    return SSB_ERR_UNSUPPORTED;
#undef SSB_SXV
}

template <typename T, int S>
static int launch_stream_taps(const SxArgs& a, int n_tokens, bool pdl, cudaStream_t stream) {
    if (a.conv_w == nullptr) return launch_stream_vec<T, S, 0>(a, n_tokens, pdl, stream);
    if (a.taps == 1) return launch_stream_vec<T, S, 1>(a, n_tokens, pdl, stream);
    if (a.taps == 2) return launch_stream_vec<T, S, 2>(a, n_tokens, pdl, stream);
    if (a.taps == 3) return launch_stream_vec<T, S, 3>(a, n_tokens, pdl, stream);
    return launch_stream_vec<T, S, 4>(a, n_tokens, pdl, stream);
}

// See SxArgs.  branch null: no write (mix, out_w and dst are not read).  norm_w null: out is float32 and gets u.
SSB_API int ssb_stream_cross(const float* src, int n_src, long long plane, float* branch, int clear, const float* mix,
                             const float* out_w, float* dst, const float* in_w, const float* norm_w, float eps, void* out,
                             int out_dtype, const float* conv_w, float* tail, const int* slot, int taps, int n_tokens,
                             int width, int streams, int pdl, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const size_t smem = norm_w != nullptr ? (size_t)width * sizeof(float) : 0;
    if (width <= 0 || smem > 200 * 1024 || streams < 1 || streams > SX_MAX_STREAMS || (n_src != 1 && n_src != streams) ||
        out == nullptr || (branch != nullptr && (mix == nullptr || out_w == nullptr)) ||
        (conv_w != nullptr && (norm_w == nullptr || taps < 1 || taps > SX_MAX_TAPS || slot == nullptr || (taps > 1 && tail == nullptr))) ||
        (norm_w == nullptr && out_dtype != SSB_F32) || (dst != nullptr && dst == src && n_src != streams))
        return SSB_ERR_BAD_SIZE;
    SxArgs a;
    a.src = src; a.n_src = n_src; a.plane = plane; a.branch = branch; a.clear = clear; a.mix = mix; a.out_w = out_w;
    a.dst = branch != nullptr ? dst : nullptr;
    a.in_w = in_w; a.norm_w = norm_w; a.eps = eps; a.out = out; a.conv_w = conv_w; a.tail = tail; a.slot = slot;
    a.taps = taps; a.width = width; a.streams = streams;
    int rc;
    const uintptr_t align = (uintptr_t)src | (uintptr_t)branch | (uintptr_t)a.dst | (uintptr_t)norm_w | (uintptr_t)out;
    const uintptr_t conv_align = conv_w == nullptr ? 0 : (uintptr_t)conv_w | (taps > 1 ? (uintptr_t)tail : 0);
    if (width % 4 == 0 && width <= (conv_w != nullptr ? 4096 : 8192) && streams <= 4 && ((align | conv_align) & 15) == 0 &&
        plane % 4 == 0 && (conv_w == nullptr || taps <= SX_VEC_TAPS)) {
        const bool chain = pdl != 0;
#define SSB_SXT(S) rc = out_dtype == SSB_F32 ? launch_stream_taps<float, S>(a, n_tokens, chain, stream) \
                                             : launch_stream_taps<bf16, S>(a, n_tokens, chain, stream)
        if (out_dtype != SSB_F32 && out_dtype != SSB_BF16) return SSB_ERR_BAD_DTYPE;
        if (streams == 1) SSB_SXT(1); else if (streams == 2) SSB_SXT(2); else if (streams == 3) SSB_SXT(3); else SSB_SXT(4);
#undef SSB_SXT
        return rc ? rc : ssb_launch_status();
    }
    const int threads = 256;
#define SSB_SX(TYPE, SM)                                                                                             \
    {                                                                                                                \
        auto kern = stream_cross_kernel<TYPE, SM>;                                                                   \
        if (smem > 48 * 1024) {                                                                                      \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        rc = ssb_launch(kern, dim3(n_tokens), dim3(threads), smem, stream, pdl != 0, a);                             \
    }
#define SSB_SX_S(TYPE)                                                                                               \
    if (streams <= 2) SSB_SX(TYPE, 2) else if (streams <= 4) SSB_SX(TYPE, 4) else if (streams <= 8) SSB_SX(TYPE, 8)  \
    else SSB_SX(TYPE, 16)
    if (out_dtype == SSB_F32) { SSB_SX_S(float) }
    else if (out_dtype == SSB_BF16) { SSB_SX_S(bf16) }
    else return SSB_ERR_BAD_DTYPE;
#undef SSB_SX_S
#undef SSB_SX
    return rc ? rc : ssb_launch_status();
}
