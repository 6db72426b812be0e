// Real-gated linear recurrent unit on mixed batches — include/atoma_hybrid.h (atoma_lru_gates, atoma_linear_scan).
//
// The unit keeps one float per channel: S <- a S + sqrt(1 - a^2) i u, where the decay a and the input gate i come from the filtered
// input u through block-diagonal matrices.  Two operators:
//   - the gates: two products per diagonal block whose epilogue forms, in float32, the decay and the gated input of every token and
//     channel — everything transcendental happens once, in parallel over tokens (bfloat16: tc::gemm_kernel with an epilogue of its
//     own; float32: FMA tiles, k ascending),
//   - the scan: a first-order linear recurrence over those two float32 arrays, times the activated gate branch.  Portions of at least
//     4 x 32 tokens run as a blocked scan (the recurrence composes: (a2, b2) o (a1, b1) = (a2 a1, a2 b1 + b2)), shorter ones and
//     decoded tokens walk in order.
#include "common.cuh"
#include "hybrid_common.cuh"
#include "tc_products.cuh"

#include "atoma_hybrid.h"

#include <algorithm>

namespace atoma {

extern int g_hybrid_debug;   // bit 0: float32 FMA products everywhere; bit 2: scans in token order whatever the portion

namespace {

using namespace hybrid;

// ---------------------------------------------------------------------------------------------
// gates, float32 FMA tiles: 64 tokens x 64 channels of one diagonal block, both products, k ascending
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) lru_gates_kernel(const atoma_lru_gates_args a, int n) {
    __shared__ float us[16][65], rs[16][65], is[16][65];
    pdl_launch_dependents();
    pdl_wait();
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, M = static_cast<int>(a.T);
    const int64_t blk = blockIdx.z;
    const T *u = static_cast<const T *>(a.u) + blk * n;
    const T *wr = static_cast<const T *>(a.w) + blk * 2 * n * n, *wi = wr + static_cast<int64_t>(n) * n;
    float ar[4][4] = {}, ai[4][4] = {};
    for (int k0 = 0; k0 < n; k0 += 16) {
        for (int i = threadIdx.x; i < 64 * 16; i += 256) {
            const int r = i / 16, k = i % 16;
            const bool kin = k0 + k < n, nin = n0 + r < n;
            us[k][r] = (kin && m0 + r < M) ? to_f(u[static_cast<int64_t>(m0 + r) * a.ld_u + k0 + k]) : 0.f;
            rs[k][r] = (kin && nin) ? to_f(wr[static_cast<int64_t>(n0 + r) * n + k0 + k]) : 0.f;
            is[k][r] = (kin && nin) ? to_f(wi[static_cast<int64_t>(n0 + r) * n + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            float uv[4], rv[4], iv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                uv[i] = us[k][ty * 4 + i];
                rv[i] = rs[k][tx * 4 + i];
                iv[i] = is[k][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    ar[i][j] = fmaf(uv[i], rv[j], ar[i][j]);
                    ai[i][j] = fmaf(uv[i], iv[j], ai[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int m = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
            if (m >= M || c >= n) continue;
            const int64_t ch = blk * n + c, o = static_cast<int64_t>(m) * a.channels + ch;
            float d, in;
            tc::lru_gates(ar[i][j] + a.bias_r[ch], ai[i][j] + a.bias_i[ch], a.rate[ch], to_f(u[static_cast<int64_t>(m) * a.ld_u + c]), d, in);
            a.decay[o] = d;
            a.input[o] = in;
        }
}

// ---------------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------------
constexpr int kBatch = 8;     // tokens whose loads are issued together before any of them is used

template <typename T>
__global__ void __launch_bounds__(128) linear_scan_seq_kernel(const atoma_linear_scan_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.y, C = static_cast<int>(a.channels);
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int t0 = a.query_start[b], t1 = a.query_start[b + 1];
    if (t1 <= t0) return;
    float *st = a.state + static_cast<int64_t>(a.state_slots[b]) * a.state_stride + c;
    float s = a.context_lens[b] > 0 ? *st : 0.f;
    const float gb = a.gate_bias ? a.gate_bias[c] : 0.f;
    const T *gate = static_cast<const T *>(a.gate);
    T *out = static_cast<T *>(a.out);
    for (int t = t0; t < t1; t += kBatch) {
        float d[kBatch], x[kBatch];
        T g[kBatch];
#pragma unroll
        for (int i = 0; i < kBatch; ++i)
            if (t + i < t1) {
                const int64_t o = static_cast<int64_t>(t + i) * C + c;
                d[i] = a.decay[o];
                x[i] = a.input[o];
                g[i] = gate[static_cast<int64_t>(t + i) * a.ld_gate + c];
            }
#pragma unroll
        for (int i = 0; i < kBatch; ++i)
            if (t + i < t1) {
                s = fmaf(d[i], s, x[i]);
                out[static_cast<int64_t>(t + i) * C + c] = from_f<T>(s * glu_act(to_f(g[i]) + gb, a.act));
            }
    }
    *st = s;
}

// A CTA owns 32 channels of one sequence; its kSeg segment rows each fold a contiguous run of tokens, the summaries are chained in
// order, and each row then replays its run from its true start value and writes the gated output.
constexpr int kSeg = 32;
template <typename T>
__global__ void __launch_bounds__(32 * kSeg) linear_scan_blocked_kernel(const atoma_linear_scan_args a) {
    __shared__ float sa[kSeg][33], sb[kSeg][33];
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.y, C = static_cast<int>(a.channels);
    const int lane = threadIdx.x, seg = threadIdx.y;
    const int c = blockIdx.x * 32 + lane;
    const int t0 = a.query_start[b], n = a.query_start[b + 1] - t0;
    if (n <= 0) return;
    const bool live = c < C;
    const int per = (n + kSeg - 1) / kSeg;
    const int lo = t0 + min(n, seg * per), hi = t0 + min(n, (seg + 1) * per);
    float A = 1.f, B = 0.f;
    if (live)
        for (int t = lo; t < hi; t += kBatch) {
            float d[kBatch], x[kBatch];
#pragma unroll
            for (int i = 0; i < kBatch; ++i)
                if (t + i < hi) {
                    const int64_t o = static_cast<int64_t>(t + i) * C + c;
                    d[i] = a.decay[o];
                    x[i] = a.input[o];
                }
#pragma unroll
            for (int i = 0; i < kBatch; ++i)
                if (t + i < hi) {
                    A *= d[i];
                    B = fmaf(d[i], B, x[i]);
                }
        }
    sa[seg][lane] = A;
    sb[seg][lane] = B;
    __syncthreads();
    float *st = a.state + (live ? static_cast<int64_t>(a.state_slots[b]) * a.state_stride + c : 0);
    float s = (live && a.context_lens[b] > 0) ? *st : 0.f;
    for (int k = 0; k < seg; ++k) s = fmaf(sa[k][lane], s, sb[k][lane]);
    __syncthreads();          // every row has read the carried state before the last one replaces it
    if (!live) return;
    const float gb = a.gate_bias ? a.gate_bias[c] : 0.f;
    const T *gate = static_cast<const T *>(a.gate);
    T *out = static_cast<T *>(a.out);
    for (int t = lo; t < hi; t += kBatch) {
        float d[kBatch], x[kBatch];
        T g[kBatch];
#pragma unroll
        for (int i = 0; i < kBatch; ++i)
            if (t + i < hi) {
                const int64_t o = static_cast<int64_t>(t + i) * C + c;
                d[i] = a.decay[o];
                x[i] = a.input[o];
                g[i] = gate[static_cast<int64_t>(t + i) * a.ld_gate + c];
            }
#pragma unroll
        for (int i = 0; i < kBatch; ++i)
            if (t + i < hi) {
                s = fmaf(d[i], s, x[i]);
                out[static_cast<int64_t>(t + i) * C + c] = from_f<T>(s * glu_act(to_f(g[i]) + gb, a.act));
            }
    }
    if (seg == kSeg - 1) *st = s;     // an empty last run carries its start value, which is the portion's end
}

}  // namespace

#define HYB_DISPATCH(dtype, CALL) ((dtype) == ATOMA_DTYPE_BF16 ? CALL(__nv_bfloat16) : CALL(float))

bool hyb_lru_gates(const atoma_lru_gates_args &a, cudaStream_t stream) {
    if (a.T <= 0) return true;
    if (!hybrid::known_dtype(a.dtype, "atoma_lru_gates")) return false;
    if (!a.u || !a.w || !a.bias_r || !a.bias_i || !a.rate || !a.decay || !a.input || a.blocks <= 0 || a.channels <= 0 || a.channels % a.blocks ||
        a.ld_u < a.channels) {
        set_status(kErrInvalidArg, "atoma_lru_gates: null argument, or %lld channels in %lld blocks", static_cast<long long>(a.channels),
                   static_cast<long long>(a.blocks));
        return false;
    }
    const int64_t n = a.channels / a.blocks;
    const dim3 grid(static_cast<unsigned>((n + 63) / 64), static_cast<unsigned>((a.T + 63) / 64), static_cast<unsigned>(a.blocks));
    if (a.dtype == ATOMA_DTYPE_BF16 && !(g_hybrid_debug & 1)) {
        tc::GemmArgs p{};
        p.a = a.u, p.lda = a.ld_u, p.a_zs = n;
        p.b = static_cast<const __nv_bfloat16 *>(a.w), p.b_zs = 2 * n * n, p.b_ks = 1, p.b_ns = n;
        p.M = static_cast<int>(a.T), p.N = p.K = static_cast<int>(n);
        p.bias_r = a.bias_r, p.bias_i = a.bias_i, p.rate = a.rate, p.decay = a.decay, p.input = a.input, p.ld_state = a.channels;
        return hybrid::launched(launch_ex(tc::gemm_kernel<__nv_bfloat16, __nv_bfloat16, tc::kEpiLru>, grid, dim3(128), 0, stream, p), "tc::gemm_kernel<lru>");
    }
#define CALL(TT) launch_ex(lru_gates_kernel<TT>, grid, dim3(256), 0, stream, a, static_cast<int>(n))
    return hybrid::launched(HYB_DISPATCH(a.dtype, CALL), "lru_gates_kernel");
#undef CALL
}

bool hyb_linear_scan(const atoma_linear_scan_args &a, cudaStream_t stream) {
    if (a.T <= 0 || a.B <= 0) return true;
    if (!hybrid::known_dtype(a.dtype, "atoma_linear_scan")) return false;
    if (!a.decay || !a.input || !a.gate || !a.state || !a.state_slots || !a.query_start || !a.context_lens || !a.out || a.channels <= 0 ||
        a.ld_gate < a.channels || a.state_stride < a.channels || a.act < 0 || a.act > 2) {
        set_status(kErrInvalidArg, "atoma_linear_scan: null argument, a row shorter than the channels, or unknown activation %d", a.act);
        return false;
    }
    if (a.max_query_len >= 4 * kSeg && !(g_hybrid_debug & 4)) {
        const dim3 grid(static_cast<unsigned>((a.channels + 31) / 32), static_cast<unsigned>(a.B));
#define CALL(TT) launch_ex(linear_scan_blocked_kernel<TT>, grid, dim3(32, kSeg), 0, stream, a)
        return hybrid::launched(HYB_DISPATCH(a.dtype, CALL), "linear_scan_blocked_kernel");
#undef CALL
    }
    const dim3 grid(static_cast<unsigned>((a.channels + 127) / 128), static_cast<unsigned>(a.B));
#define CALL(TT) launch_ex(linear_scan_seq_kernel<TT>, grid, dim3(128), 0, stream, a)
    return hybrid::launched(HYB_DISPATCH(a.dtype, CALL), "linear_scan_seq_kernel");
#undef CALL
}

}  // namespace atoma

using namespace atoma;

extern "C" void atoma_lru_gates(const atoma_lru_gates_args *args, atoma_stream_t stream) {
    clear_status();
    if (!args) {
        set_status(kErrInvalidArg, "atoma_lru_gates: args is NULL");
        return;
    }
    hyb_lru_gates(*args, static_cast<cudaStream_t>(stream));
}

extern "C" void atoma_linear_scan(const atoma_linear_scan_args *args, atoma_stream_t stream) {
    clear_status();
    if (!args) {
        set_status(kErrInvalidArg, "atoma_linear_scan: args is NULL");
        return;
    }
    hyb_linear_scan(*args, static_cast<cudaStream_t>(stream));
}
