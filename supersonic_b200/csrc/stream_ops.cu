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
    const float* conv_w;         // [width][taps], or null: no convolution behind the norm
    float* tail;                 // [slots][taps - 1][width] the last taps - 1 normed rows, oldest first
    const int* slot;             // [tokens]
    int taps, width, streams;
};

// One block per token; u's row waits in shared memory for its sum of squares, which is taken in a fixed order.
// SM: an upper bound of the number of streams (the loops over them are unrolled).
template <typename T, int SM>
__global__ void stream_cross_kernel(const SxArgs a) {
    extern __shared__ float sx_row[];
    __shared__ float red[32];
    __shared__ float c_mix[SM * SM], c_out[SM], c_in[SM];
    const int tid = threadIdx.x, nt = blockDim.x, S = a.streams, W = a.width;
    const bool writes = a.branch != nullptr;
    ssb_pdl_launch_dependents();
    // the coefficients are weights: no kernel of a step writes them
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
            if (a.clear) br[c] = 0.f;
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
        if (a.norm_w == nullptr) {
            reinterpret_cast<float*>(a.out)[t * W + c] = u;
            continue;
        }
        sx_row[c] = u;
        sq = fmaf(u, u, sq);
    }
    if (a.norm_w == nullptr) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if ((tid & 31) == 0) red[tid >> 5] = sq;
    __syncthreads();
    float total = 0.f;
    for (int w = 0; w < nt / 32; ++w) total += red[w];
    const float inv = 1.0f / sqrtf(total / (float)W + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + t * W;
    if (a.conv_w == nullptr) {
        for (int c = tid; c < W; c += nt) out[c] = ssb_from_float<T>(sx_row[c] * inv * a.norm_w[c]);
        return;
    }
    const int slot = a.slot[t], back = a.taps - 1;
    for (int c = tid; c < W; c += nt) {
        const float n = sx_row[c] * inv * a.norm_w[c];
        const float* w = a.conv_w + (size_t)c * a.taps;
        float acc = 0.f;
        if (slot >= 0 && back > 0) {                       // the kept rows move down by one place
            float* keep = a.tail + (size_t)slot * back * W + c;
            for (int j = 0; j < back; ++j) {
                const float v = keep[(size_t)j * W];
                acc = fmaf(w[j], v, acc);
                if (j > 0) keep[(size_t)(j - 1) * W] = v;
            }
            keep[(size_t)(back - 1) * W] = n;
        }
        out[c] = ssb_from_float<T>(fmaf(w[back], n, acc));
    }
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
    // few tokens: a block's latency is the step's, so more threads share a row
    const int threads = n_tokens <= 148 && width >= 1024 ? 512 : 256;
    int rc;
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
