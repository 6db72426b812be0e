// Residual update of POST-NORM decoder blocks — include/atoma_hybrid.h (atoma_postnorm_residual).
//
// The stream is normed after every sum, x <- norm(alpha x + sublayer), and the sublayers read it as it is.  After a layer the stream
// may become a weighted average over DEPTH: of the embedding output and of every layer's result so far, which are kept as float32
// rows [layer][token][width] for the step.  One CTA per token does the sum (with the token's routed experts' rows), the norm, the
// write of the layer's row, the average, and the copy in the activation format that the next sublayer's projections read.
// A second form norms the sublayer's result instead of the sum and adds it to the stream (norm_branch).
// Everything is float32; rows are reduced in an order that depends on the row alone.
#include "common.cuh"
#include "hybrid_common.cuh"

#include "atoma_hybrid.h"

namespace atoma {
namespace {

using namespace hybrid;

constexpr int kMaxTop = 64;       // router choices per token
constexpr int kDepthBatch = 4;    // depth rows whose loads are in flight together

template <typename T, bool VEC>
struct Quad;   // four consecutive channels (VEC) or one
template <typename T>
struct Quad<T, true> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float *p, float (&v)[4]) {
        const float4 x = *reinterpret_cast<const float4 *>(p);
        v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
    }
    static __device__ __forceinline__ void load(const __nv_bfloat16 *p, float (&v)[4]) {
        const uint2 x = *reinterpret_cast<const uint2 *>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&x.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&x.y));
        v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
    }
    static __device__ __forceinline__ void store(float *p, const float (&v)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, const float (&v)[4]) {
        uint2 x;
        x.x = pack2<__nv_bfloat16>(v[0], v[1]);
        x.y = pack2<__nv_bfloat16>(v[2], v[3]);
        *reinterpret_cast<uint2 *>(p) = x;
    }
};
template <typename T>
struct Quad<T, false> {
    static constexpr int N = 1;
    template <typename S>
    static __device__ __forceinline__ void load(const S *p, float (&v)[1]) { v[0] = to_f(*p); }
    template <typename S>
    static __device__ __forceinline__ void store(S *p, const float (&v)[1]) { *p = from_f<S>(v[0]); }
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(kRowThreads) postnorm_residual_kernel(const atoma_postnorm_args a) {
    using Q = Quad<T, VEC>;
    constexpr int C = Q::N;
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    __shared__ int64_t erow[kMaxTop];       // offset of the pair's expert row, -1: none
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int W = static_cast<int>(a.width);
    const int top = a.expert_out ? static_cast<int>(a.top) : 0;
    for (int k = threadIdx.x; k < top; k += blockDim.x) {
        const bool there = !a.top_expert || a.top_expert[t * top + k] >= 0;
        erow[k] = there ? static_cast<int64_t>(a.pair_row[t * top + k]) * W : -1;
    }
    if (top > 0) __syncthreads();
    const T *y = a.y ? static_cast<const T *>(a.y) + t * W : nullptr;
    const T *eo = static_cast<const T *>(a.expert_out);
    float *x = a.x + t * W;
    float ss = 0.f;
    for (int c = C * threadIdx.x; c < W; c += C * blockDim.x) {
        float v[C], s[C];
        if (a.norm_branch) {
#pragma unroll
            for (int i = 0; i < C; ++i) v[i] = 0.f;
            if (y) {
                Q::load(y + c, s);
#pragma unroll
                for (int i = 0; i < C; ++i) v[i] = a.y_scale * s[i];
            }
            if (a.y_bias) {
                Q::load(a.y_bias + c, s);
#pragma unroll
                for (int i = 0; i < C; ++i) v[i] += s[i];
            }
        } else {
            Q::load(x + c, v);
#pragma unroll
            for (int i = 0; i < C; ++i) v[i] *= a.alpha;
            if (y) {
                Q::load(y + c, s);
#pragma unroll
                for (int i = 0; i < C; ++i) v[i] += s[i];
            }
        }
        for (int k = 0; k < top; ++k) {
            if (erow[k] < 0) continue;
            Q::load(eo + erow[k] + c, s);
#pragma unroll
            for (int i = 0; i < C; ++i) v[i] += s[i];
        }
#pragma unroll
        for (int i = 0; i < C; ++i) {
            row[c + i] = v[i];
            ss = fmaf(v[i], v[i], ss);
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + a.eps);
    const int64_t plane = a.T * W;
    const int nd = static_cast<int>(a.depth_n);
    T *h = a.h ? static_cast<T *>(a.h) + t * W : nullptr;
    // a thread reads back the channels of `row` that it wrote itself
    for (int c = C * threadIdx.x; c < W; c += C * blockDim.x) {
        float n[C], w[C];
        Q::load(a.w_norm + c, w);
#pragma unroll
        for (int i = 0; i < C; ++i) n[i] = row[c + i] * inv * (a.weight_offset + w[i]);
        if (a.norm_branch) {
            float s[C];
            Q::load(x + c, s);
#pragma unroll
            for (int i = 0; i < C; ++i) n[i] = fmaf(a.branch_scale, n[i], a.alpha * s[i]);
        }
        if (nd > 0) {
            float *d = a.depth + t * W + c;
            Q::store(d + (nd - 1) * plane, n);
            if (a.depth_w) {
                float acc[C];
#pragma unroll
                for (int i = 0; i < C; ++i) acc[i] = 0.f;
                for (int j0 = 0; j0 + 1 < nd; j0 += kDepthBatch) {
                    float r[kDepthBatch][C];
#pragma unroll
                    for (int u = 0; u < kDepthBatch; ++u)
                        if (j0 + u + 1 < nd) Q::load(d + (j0 + u) * plane, r[u]);
#pragma unroll
                    for (int u = 0; u < kDepthBatch; ++u)
                        if (j0 + u + 1 < nd) {
                            const float dw = a.depth_w[j0 + u];
#pragma unroll
                            for (int i = 0; i < C; ++i) acc[i] = fmaf(dw, r[u][i], acc[i]);
                        }
                }
                const float dw = a.depth_w[nd - 1];
#pragma unroll
                for (int i = 0; i < C; ++i) n[i] = fmaf(dw, n[i], acc[i]);
            }
        }
        Q::store(x + c, n);
        if (h) Q::store(h + c, n);
        if (a.trace) Q::store(a.trace + t * W + c, n);
    }
}

}  // namespace

bool hyb_postnorm_residual(const atoma_postnorm_args &a, cudaStream_t stream) {
    if (a.T <= 0) return true;
    if (!hybrid::known_dtype(a.dtype, "atoma_postnorm_residual")) return false;
    if (!a.x || !a.w_norm || a.width <= 0 || a.depth_n < 0 || (a.depth_n > 0 && !a.depth) ||
        (a.expert_out && (!a.pair_row || a.top <= 0 || a.top > kMaxTop))) {
        set_status(kErrInvalidArg, "atoma_postnorm_residual: null or inconsistent arguments (at most %d choices per token)", kMaxTop);
        return false;
    }
    const size_t smem = static_cast<size_t>(a.width) * 4;
    if (smem > 200 * 1024) {
        set_status(kErrUnsupported, "atoma_postnorm_residual: a width of %lld exceeds shared memory", static_cast<long long>(a.width));
        return false;
    }
    auto al = [](const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = a.width % 4 == 0 && al(a.x) && al(a.y) && al(a.expert_out) && al(a.w_norm) && al(a.y_bias) && al(a.depth) && al(a.h) && al(a.trace);
    cudaError_t e;
#define CASE(TT, V)                                                                                                                       \
    {                                                                                                                                     \
        if (smem > 48 * 1024) cudaFuncSetAttribute(postnorm_residual_kernel<TT, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
        e = launch_ex(postnorm_residual_kernel<TT, V>, dim3(static_cast<unsigned>(a.T)), dim3(kRowThreads), smem, stream, a);             \
    }
    if (a.dtype == ATOMA_DTYPE_BF16) {
        if (vec) CASE(__nv_bfloat16, true) else CASE(__nv_bfloat16, false)
    } else {
        if (vec) CASE(float, true) else CASE(float, false)
    }
#undef CASE
    return hybrid::launched(e, "postnorm_residual_kernel");
}

}  // namespace atoma

using namespace atoma;

extern "C" void atoma_postnorm_residual(const atoma_postnorm_args *args, atoma_stream_t stream) {
    clear_status();
    if (!args) {
        set_status(kErrInvalidArg, "atoma_postnorm_residual: args is NULL");
        return;
    }
    hyb_postnorm_residual(*args, static_cast<cudaStream_t>(stream));
}
