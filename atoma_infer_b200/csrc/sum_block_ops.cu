// Operators around differential attention and the state-space recurrence — include/atoma_hybrid.h (atoma_embed_pairs,
// atoma_differential_combine, atoma_gate_groupnorm).
//
// All three are row operators bound by memory: the embedding with its second, pair-indexed table (and the copy the first layer reads),
// the weighted difference of a head's two softmax maps at unit root mean square, and the gate and grouped norm behind a recurrence's
// float32 read-out.  Statistics are float32 and are reduced in an order that depends on the row alone.
#include "common.cuh"
#include "hybrid_common.cuh"

#include "atoma_hybrid.h"

#include <algorithm>

namespace atoma {
namespace {

using namespace hybrid;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
    return v;
}

// N consecutive elements of a row: one access when N > 1 (the host checked alignment).
template <int N>
__device__ __forceinline__ void load_n(const float *p, float (&v)[N]) {
    if constexpr (N % 4 == 0) {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const float4 x = *reinterpret_cast<const float4 *>(p + i);
            v[i] = x.x, v[i + 1] = x.y, v[i + 2] = x.z, v[i + 3] = x.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = p[i];
    }
}
template <int N>
__device__ __forceinline__ void load_n(const __nv_bfloat16 *p, float (&v)[N]) {
    if constexpr (N == 4) {
        const uint2 x = *reinterpret_cast<const uint2 *>(p);
        const uint32_t u[2] = {x.x, x.y};
#pragma unroll
        for (int i = 0; i < 2; ++i) v[2 * i] = __uint_as_float(u[i] << 16), v[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = to_f(p[i]);
    }
}
template <int N>
__device__ __forceinline__ void store_n(float *p, const float (&v)[N]) {
    if constexpr (N == 4) *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else
#pragma unroll
        for (int i = 0; i < N; ++i) p[i] = v[i];
}
template <int N>
__device__ __forceinline__ void store_n(__nv_bfloat16 *p, const float (&v)[N]) {
    if constexpr (N == 4) {
        uint2 x;
        x.x = pack2<__nv_bfloat16>(v[0], v[1]);
        x.y = pack2<__nv_bfloat16>(v[2], v[3]);
        *reinterpret_cast<uint2 *>(p) = x;
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) p[i] = from_f<__nv_bfloat16>(v[i]);
    }
}

struct EmbedPairs {
    const uint32_t *tokens;
    const int32_t *token_seq, *query_start, *prev_tokens;
    const void *table, *pair_table;
    int64_t buckets, mul_prev, mul_cur;
    float *x;
    void *h;
    int width;
    int64_t vocab;
};

template <typename T, int N>
__global__ void __launch_bounds__(128) embed_pairs_kernel(const EmbedPairs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int64_t tok = min(static_cast<int64_t>(a.tokens[t]), a.vocab - 1);
    const T *e = static_cast<const T *>(a.table) + tok * a.width;
    const T *e2 = nullptr;
    if (a.pair_table) {
        const int b = a.token_seq[t];
        const int64_t before = t > a.query_start[b] ? static_cast<int64_t>(a.tokens[t - 1]) : static_cast<int64_t>(a.prev_tokens[b]);
        int64_t row = a.buckets;
        if (before >= 0) {
            row = (before * a.mul_prev + static_cast<int64_t>(a.tokens[t]) * a.mul_cur) % a.buckets;
            if (row < 0) row += a.buckets;
        }
        e2 = static_cast<const T *>(a.pair_table) + row * a.width;
    }
    float *x = a.x + t * a.width;
    T *h = a.h ? static_cast<T *>(a.h) + t * a.width : nullptr;
    for (int c = N * threadIdx.x; c < a.width; c += N * blockDim.x) {
        float v[N], w[N];
        load_n<N>(e + c, v);
        if (e2) {
            load_n<N>(e2 + c, w);
#pragma unroll
            for (int i = 0; i < N; ++i) v[i] += w[i];
        }
        store_n<N>(x + c, v);
        if (h) store_n<N>(h + c, v);
    }
}

// One warp per (token, head).
template <typename T, int N>
__global__ void __launch_bounds__(256) differential_combine_kernel(const T *__restrict__ maps, T *__restrict__ out, int64_t rows, int H, int rep, int V,
                                                                   float lambda, float gain, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t wid = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (wid >= rows) return;
    const int lane = threadIdx.x & 31;
    const int64_t t = wid / H;
    const int h = static_cast<int>(wid % H), g = h / rep, r = h % rep;
    const T *p1 = maps + ((t * 2 * H) + 2 * g * rep + r) * V, *p2 = p1 + static_cast<int64_t>(rep) * V;
    T *o = out + wid * V;
    float ss = 0.f;
    for (int c = N * lane; c < V; c += 32 * N) {
        float a1[N], a2[N];
        load_n<N>(p1 + c, a1);
        load_n<N>(p2 + c, a2);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const float d = fmaf(-lambda, a2[i], a1[i]);
            ss = fmaf(d, d, ss);
        }
    }
    const float f = gain / sqrtf(warp_sum(ss) / static_cast<float>(V) + eps);
    for (int c = N * lane; c < V; c += 32 * N) {   // the second read hits the first-level cache
        float a1[N], a2[N];
        load_n<N>(p1 + c, a1);
        load_n<N>(p2 + c, a2);
#pragma unroll
        for (int i = 0; i < N; ++i) a1[i] = fmaf(-lambda, a2[i], a1[i]) * f;
        store_n<N>(o + c, a1);
    }
}

// One CTA per token; the gated row stays in shared memory between the statistics and the store.  Few parts: several
// warps each; many: the warps take them in turn.
template <typename T, int N>
__global__ void __launch_bounds__(kRowThreads) gate_groupnorm_kernel(const float *__restrict__ o, const T *__restrict__ gate, int64_t ld_gate,
                                                                     const float *__restrict__ weight, T *__restrict__ out, int64_t ld_out, int n, int parts,
                                                                     int zero_before, int zero_after, float eps) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const float *src = o + t * n;
    const T *gt = gate + t * ld_gate;
    T *dst = out + t * ld_out;
    const int per = n / parts, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    for (int c = threadIdx.x; c < zero_before; c += blockDim.x) dst[c - zero_before] = from_f<T>(0.f);
    for (int c = threadIdx.x; c < zero_after; c += blockDim.x) dst[n + c] = from_f<T>(0.f);
    auto gated = [&](int c, float (&u)[N]) {
        float z[N];
        load_n<N>(src + c, u);
        load_n<N>(gt + c, z);
#pragma unroll
        for (int i = 0; i < N; ++i) u[i] *= silu(z[i]);
    };
    auto finish = [&](int c, float inv) {
        float w[N], v[N];
        load_n<N>(weight + c, w);
        load_n<N>(row + c, v);
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = v[i] * inv * w[i];
        store_n<N>(dst + c, v);
    };
    const int wpp = max(1, nwarp / parts);         // warps per part; more than one: every part has its warps, in one go
    for (int p = warp / wpp; p < (wpp > 1 ? nwarp / wpp : parts); p += nwarp / wpp) {
        const int c0 = p * per, c1 = p < parts ? c0 + per : c0;
        const int first = c0 + N * (lane + 32 * (warp % wpp)), step = 32 * N * wpp;
        float ss = 0.f;
        for (int c = first; c < c1; c += step) {
            float u[N];
            gated(c, u);
            store_n<N>(row + c, u);
#pragma unroll
            for (int i = 0; i < N; ++i) ss = fmaf(u[i], u[i], ss);
        }
        ss = warp_sum(ss);
        if (wpp > 1) {
            if (lane == 0) red[warp] = ss;
            __syncthreads();                       // every warp makes exactly one pass here
            ss = 0.f;
            for (int w = 0; w < wpp; ++w) ss += red[warp / wpp * wpp + w];
        }
        const float inv = 1.0f / sqrtf(ss / static_cast<float>(per) + eps);
        for (int c = first; c < c1; c += step) finish(c, inv);   // what this thread stored itself
    }
}

bool aligned16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

bool hyb_embed_pairs(const uint32_t *tokens, const int32_t *token_seq, const int32_t *query_start, const int32_t *prev_tokens, const void *table,
                     const void *pair_table, int64_t buckets, int64_t mul_prev, int64_t mul_cur, float *x, void *h, int64_t T, int64_t width,
                     int64_t vocab, uint32_t dtype, cudaStream_t stream) {
    if (T <= 0) return true;
    if (!hybrid::known_dtype(dtype, "atoma_embed_pairs")) return false;
    if (!tokens || !table || !x || width <= 0 || vocab <= 0 || (pair_table && (!token_seq || !query_start || !prev_tokens || buckets <= 0))) {
        set_status(kErrInvalidArg, "atoma_embed_pairs: null argument or empty shape");
        return false;
    }
    const EmbedPairs a{tokens, token_seq, query_start, prev_tokens, table, pair_table, buckets, mul_prev, mul_cur, x, h, static_cast<int>(width), vocab};
    const bool vec = width % 4 == 0 && aligned16(table) && aligned16(pair_table) && aligned16(x) && aligned16(h);
#define CALL(TT, N) launch_ex(embed_pairs_kernel<TT, N>, dim3(static_cast<unsigned>(T)), dim3(128), 0, stream, a)
    const cudaError_t e = dtype == ATOMA_DTYPE_BF16 ? (vec ? CALL(__nv_bfloat16, 4) : CALL(__nv_bfloat16, 1)) : (vec ? CALL(float, 4) : CALL(float, 1));
#undef CALL
    return hybrid::launched(e, "embed_pairs_kernel");
}

bool hyb_differential_combine(const void *maps, void *out, int64_t T, int64_t H, int64_t G, int64_t vdim, float lambda, float gain, float eps,
                              uint32_t dtype, cudaStream_t stream) {
    if (T <= 0) return true;
    if (!hybrid::known_dtype(dtype, "atoma_differential_combine")) return false;
    if (!maps || !out || H <= 0 || G <= 0 || H % G || vdim <= 0) {
        set_status(kErrInvalidArg, "atoma_differential_combine: null argument or inconsistent head counts");
        return false;
    }
    const int64_t rows = T * H;
    const bool vec = vdim % 4 == 0 && aligned16(maps) && aligned16(out);
#define CALL(TT, N) launch_ex(differential_combine_kernel<TT, N>, dim3(static_cast<unsigned>((rows + 7) / 8)), dim3(256), 0, stream,            \
                              static_cast<const TT *>(maps), static_cast<TT *>(out), rows, static_cast<int>(H), static_cast<int>(H / G), \
                              static_cast<int>(vdim), lambda, gain, eps)
    const cudaError_t e = dtype == ATOMA_DTYPE_BF16 ? (vec ? CALL(__nv_bfloat16, 4) : CALL(__nv_bfloat16, 1)) : (vec ? CALL(float, 4) : CALL(float, 1));
#undef CALL
    return hybrid::launched(e, "differential_combine_kernel");
}

bool hyb_gate_groupnorm(const float *o, const void *gate, int64_t ld_gate, const float *weight, void *out, int64_t ld_out, int64_t T, int64_t n,
                        int64_t parts, int64_t zero_before, int64_t zero_after, float eps, uint32_t dtype, cudaStream_t stream) {
    if (T <= 0) return true;
    if (!hybrid::known_dtype(dtype, "atoma_gate_groupnorm")) return false;
    if (!o || !gate || !weight || !out || n <= 0 || parts <= 0 || n % parts || ld_gate < n || zero_before < 0 || zero_after < 0 ||
        ld_out < zero_before + n + zero_after) {
        set_status(kErrInvalidArg, "atoma_gate_groupnorm: null argument, %lld columns in %lld parts, or a row shorter than its columns",
                   static_cast<long long>(n), static_cast<long long>(parts));
        return false;
    }
    const size_t smem = static_cast<size_t>(n) * 4;
    if (smem > 200 * 1024) {
        set_status(kErrUnsupported, "atoma_gate_groupnorm: %lld columns exceed shared memory", static_cast<long long>(n));
        return false;
    }
    const int64_t es = dtype == ATOMA_DTYPE_F32 ? 4 : 2;
    const bool vec = (n / parts) % 4 == 0 && aligned16(o) && aligned16(weight) && (reinterpret_cast<uintptr_t>(gate) % (4 * es)) == 0 &&
                     (reinterpret_cast<uintptr_t>(out) % (4 * es)) == 0 && ld_gate % 4 == 0 && ld_out % 4 == 0;
    cudaError_t e;
#define CALL(TT, N)                                                                                                                              \
    {                                                                                                                                            \
        if (smem > 48 * 1024) cudaFuncSetAttribute(gate_groupnorm_kernel<TT, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);       \
        e = launch_ex(gate_groupnorm_kernel<TT, N>, dim3(static_cast<unsigned>(T)), dim3(kRowThreads), smem, stream, o, static_cast<const TT *>(gate), \
                      ld_gate, weight, static_cast<TT *>(out), ld_out, static_cast<int>(n), static_cast<int>(parts), static_cast<int>(zero_before), \
                      static_cast<int>(zero_after), eps);                                                                                         \
    }
    if (dtype == ATOMA_DTYPE_BF16) {
        if (vec) CALL(__nv_bfloat16, 4) else CALL(__nv_bfloat16, 1)
    } else {
        if (vec) CALL(float, 4) else CALL(float, 1)
    }
#undef CALL
    return hybrid::launched(e, "gate_groupnorm_kernel");
}

}  // namespace atoma

using namespace atoma;

extern "C" void atoma_embed_pairs(const uint32_t *tokens, const int32_t *token_seq, const int32_t *query_start, const int32_t *prev_tokens,
                                  const void *table, const void *pair_table, int64_t buckets, int64_t mul_prev, int64_t mul_cur, float *x, void *h,
                                  int64_t T, int64_t width, int64_t vocab, uint32_t dtype, atoma_stream_t stream) {
    clear_status();
    hyb_embed_pairs(tokens, token_seq, query_start, prev_tokens, table, pair_table, buckets, mul_prev, mul_cur, x, h, T, width, vocab, dtype,
                    static_cast<cudaStream_t>(stream));
}
extern "C" void atoma_differential_combine(const void *maps, void *out, int64_t T, int64_t H, int64_t G, int64_t vdim, float lambda, float gain,
                                           float eps, uint32_t dtype, atoma_stream_t stream) {
    clear_status();
    hyb_differential_combine(maps, out, T, H, G, vdim, lambda, gain, eps, dtype, static_cast<cudaStream_t>(stream));
}
extern "C" void atoma_gate_groupnorm(const float *o, const void *gate, int64_t ld_gate, const float *weight, void *out, int64_t ld_out, int64_t T,
                                     int64_t n, int64_t parts, int64_t zero_before, int64_t zero_after, float eps, uint32_t dtype,
                                     atoma_stream_t stream) {
    clear_status();
    hyb_gate_groupnorm(o, gate, ld_gate, weight, out, ld_out, T, n, parts, zero_before, zero_after, eps, dtype, static_cast<cudaStream_t>(stream));
}
