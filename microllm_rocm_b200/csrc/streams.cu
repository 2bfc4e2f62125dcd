// A residual stream kept as several copies ("streams") that every sublayer reads and writes through small learned
// mixtures.  X [T, S, W] fp32, S streams a token side by side.  Around a sublayer with vectors a [S], b [S], a matrix
// M [S, S] (indexed [from, to]) and a result y [T, W]:
//
//   u = sum_s a_s X_s;   y = sublayer(norm(u));   X_t <- sum_s M[s, t] X_s + b_t y        (all t at once, from the old X)
//
//   mlb_streams_mix_norm   one pass between two sublayers: the pending result y of the one before (K-split partial results
//                          are added in split order) goes into the streams in place with ITS M and b, and the next one's
//                          input norm(sum_s a_s X_s) goes out in the compute dtype.  The norm is a layer norm (`centred` 1)
//                          or an rms norm, with a weight and an optional bias.  Without y the streams stay as they are.
//                          With `rows` the pass runs for those rows only and leaves the streams alone (the final norm of
//                          a few rows: a_s = 1).
//   mlb_streams_total      sum_s X_s with a pending result taken in, in fp32 (the streams stay as they are).
//
// One CTA of a fixed size per row, the row of u kept between the passes, sums over the streams in order of their index,
// reductions in a fixed tree: a row's result depends on the row alone.
#include "common.cuh"

using namespace mlb;

MLB_DEFINE_LAST_ERROR()

namespace {

constexpr int THREADS = 256;
constexpr int MAX_STREAMS = 16;

struct StreamParams {
    float* x;                                          // [T, S, W]
    const float* y; int n_y; long long y_stride;       // pending result or null
    const float* mix;                                  // [S, S] of the pending result's sublayer
    const float* out_w;                                // [S]
    const float* in_w;                                 // [S] of the next sublayer
    const float* weight; const float* bias; int centred; float eps;
    void* normed;                                      // [rows, W]
    const int* rows;
    int S, W;
};

// sum over the partial results at one float4, eight loads in flight, added in split order
__device__ __forceinline__ float4 partial_sum4(const float* at, int n, long long stride) {
    float4 total = *reinterpret_cast<const float4*>(at);
    for (int k0 = 1; k0 < n; k0 += 8) {
        float4 part[8];
#pragma unroll
        for (int k = 0; k < 8; ++k)
            part[k] = k0 + k < n ? *reinterpret_cast<const float4*>(at + (size_t)(k0 + k) * stride) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < 8; ++k) { total.x += part[k].x; total.y += part[k].y; total.z += part[k].z; total.w += part[k].w; }
    }
    return total;
}

__device__ __forceinline__ void fma4(float s, const float4& a, float4& acc) {
    acc.x = fmaf(s, a.x, acc.x); acc.y = fmaf(s, a.y, acc.y); acc.z = fmaf(s, a.z, acc.z); acc.w = fmaf(s, a.w, acc.w);
}

template <typename OutT>
__device__ __forceinline__ void store4(OutT* dst, const float4& v) {
    if constexpr (sizeof(OutT) == 4) {
        *reinterpret_cast<float4*>(dst) = v;
    } else {
        uint2 raw;
        OutT* e = reinterpret_cast<OutT*>(&raw);
        e[0] = from_f32<OutT>(v.x); e[1] = from_f32<OutT>(v.y); e[2] = from_f32<OutT>(v.z); e[3] = from_f32<OutT>(v.w);
        *reinterpret_cast<uint2*>(dst) = raw;
    }
}

// S streams, VECS float4 a thread: rows of up to 4 * VECS * THREADS columns, a multiple of four
template <typename OutT, int S, int VECS>
__global__ void __launch_bounds__(THREADS) mix_norm_kernel(StreamParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[32];
    const int W = p.W;
    // weights are never written by a kernel: they are fetched before the wait for the predecessor
    float a[S], b[S], M[S][S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        a[s] = p.in_w[s];
        b[s] = p.y ? p.out_w[s] : 0.0f;
#pragma unroll
        for (int t = 0; t < S; ++t) M[s][t] = p.y ? p.mix[s * S + t] : 0.0f;
    }
    float4 wv[VECS], bv[VECS], u[VECS];
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        bv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < W) {
            wv[i] = *reinterpret_cast<const float4*>(p.weight + c);
            if (p.bias) bv[i] = *reinterpret_cast<const float4*>(p.bias + c);
        }
    }
    pdl_wait();
    const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
    float* const xr = p.x + row * S * W;
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= W) continue;
        float4 x[S];
#pragma unroll
        for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4*>(xr + (size_t)s * W + c);
        if (p.y) {
            const float4 y = partial_sum4(p.y + row * W + c, p.n_y, p.y_stride);
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int s = 0; s < S; ++s) fma4(M[s][t], x[s], v);
                fma4(b[t], y, v);
                if (!p.rows) *reinterpret_cast<float4*>(xr + (size_t)t * W + c) = v;
                fma4(a[t], v, u[i]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) fma4(a[s], x[s], u[i]);
        }
        sum += (u[i].x + u[i].y) + (u[i].z + u[i].w);
    }
    const float mean = p.centred ? block_sum(sum, scratch) / (float)W : 0.0f;
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c >= W) continue;
        u[i].x -= mean; u[i].y -= mean; u[i].z -= mean; u[i].w -= mean;
        sq += (u[i].x * u[i].x + u[i].y * u[i].y) + (u[i].z * u[i].z + u[i].w * u[i].w);
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)W + p.eps);
    OutT* const out = (OutT*)p.normed + (size_t)blockIdx.x * W;
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c >= W) continue;
        store4(out + c, make_float4(u[i].x * inv * wv[i].x + bv[i].x, u[i].y * inv * wv[i].y + bv[i].y,
                                    u[i].z * inv * wv[i].z + bv[i].z, u[i].w * inv * wv[i].w + bv[i].w));
    }
}

__device__ __forceinline__ float pending_at(const StreamParams& p, size_t row, int c) {
    const float* at = p.y + row * p.W + c;
    float v = at[0];
    for (int k = 1; k < p.n_y; ++k) v += at[(size_t)k * p.y_stride];
    return v;
}

// any width, up to MAX_STREAMS streams; the row of u in shared memory
template <typename OutT>
__global__ void __launch_bounds__(THREADS) mix_norm_any_kernel(StreamParams p) {
    pdl_prologue();
    extern __shared__ __align__(16) float u_s[];
    __shared__ float scratch[32];
    const int W = p.W, S = p.S;
    const size_t row = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
    float* const xr = p.x + row * S * W;
    float sum = 0.0f;
    for (int c = threadIdx.x; c < W; c += THREADS) {
        float x[MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = xr[(size_t)s * W + c];
        const float y = p.y ? pending_at(p, row, c) : 0.0f;
        float u = 0.0f;
        for (int t = 0; t < S; ++t) {
            float v = x[t];
            if (p.y) {
                v = 0.0f;
                for (int s = 0; s < S; ++s) v = fmaf(p.mix[s * S + t], x[s], v);
                v = fmaf(p.out_w[t], y, v);
                if (!p.rows) xr[(size_t)t * W + c] = v;
            }
            u = fmaf(p.in_w[t], v, u);
        }
        u_s[c] = u;
        sum += u;
    }
    const float mean = p.centred ? block_sum(sum, scratch) / (float)W : 0.0f;
    float sq = 0.0f;
    for (int c = threadIdx.x; c < W; c += THREADS) { const float d = u_s[c] - mean; sq = fmaf(d, d, sq); }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)W + p.eps);
    OutT* const out = (OutT*)p.normed + (size_t)blockIdx.x * W;
    for (int c = threadIdx.x; c < W; c += THREADS)
        out[c] = from_f32<OutT>((u_s[c] - mean) * inv * p.weight[c] + (p.bias ? p.bias[c] : 0.0f));
}

__global__ void __launch_bounds__(THREADS) total_kernel(StreamParams p, float* __restrict__ out) {
    pdl_prologue();
    const int W = p.W, S = p.S;
    const size_t row = blockIdx.x;
    const float* const xr = p.x + row * S * W;
    for (int c = threadIdx.x; c < W; c += THREADS) {
        const float y = p.y ? pending_at(p, row, c) : 0.0f;
        float total = 0.0f;
        for (int t = 0; t < S; ++t) {
            float v = xr[(size_t)t * W + c];
            if (p.y) {
                v = 0.0f;
                for (int s = 0; s < S; ++s) v = fmaf(p.mix[s * S + t], xr[(size_t)s * W + c], v);
                v = fmaf(p.out_w[t], y, v);
            }
            total += v;
        }
        out[row * W + c] = total;
    }
}

template <typename OutT, int S>
bool launch_fast(const StreamParams& p, int n, cudaStream_t stream) {
    const int vecs = (p.W / 4 + THREADS - 1) / THREADS;
    if (vecs <= 1) launch_kernel(mix_norm_kernel<OutT, S, 1>, (unsigned)n, THREADS, 0, stream, p);
    else if (vecs <= 2) launch_kernel(mix_norm_kernel<OutT, S, 2>, (unsigned)n, THREADS, 0, stream, p);
    else if (vecs <= 4) launch_kernel(mix_norm_kernel<OutT, S, 4>, (unsigned)n, THREADS, 0, stream, p);
    else return false;
    return true;
}

template <typename OutT>
int launch(const StreamParams& p, int n, cudaStream_t stream) {
    const bool fours = p.W % 4 == 0 && p.y_stride % 4 == 0 &&
                       ((uintptr_t)p.x | (uintptr_t)p.y | (uintptr_t)p.weight | (uintptr_t)p.bias | (uintptr_t)p.normed) % 16 == 0;
    if (fours) {
        bool done = false;
        if (p.S == 1) done = launch_fast<OutT, 1>(p, n, stream);
        else if (p.S == 2) done = launch_fast<OutT, 2>(p, n, stream);
        else if (p.S == 3) done = launch_fast<OutT, 3>(p, n, stream);
        else if (p.S == 4) done = launch_fast<OutT, 4>(p, n, stream);
        if (done) return check_launch("streams_mix_norm");
    }
    const size_t smem = (size_t)p.W * sizeof(float);
    if (smem > 200 * 1024) return fail(MLB_UNSUPPORTED_SIZE, "streams_mix_norm: a row of %d floats does not fit shared memory", p.W);
    if (smem > 48 * 1024) {
        static bool raised[MAX_DEVICES] = {false};
        if (!raised[device_index()]) {
            if (cudaFuncSetAttribute(mix_norm_any_kernel<OutT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
                return fail(MLB_CUDA_ERROR, "streams_mix_norm: cannot raise the shared-memory limit");
            raised[device_index()] = true;
        }
    }
    launch_kernel(mix_norm_any_kernel<OutT>, (unsigned)n, THREADS, smem, stream, p);
    return check_launch("streams_mix_norm");
}

}  // namespace

MLB_EXPORT int mlb_streams_max() { return MAX_STREAMS; }

// n: rows to run (the rows of X, or the length of `rows`)
MLB_EXPORT int mlb_streams_mix_norm(float* x, const float* y, int n_y, long long y_stride, const float* mix, const float* out_w,
                                    const float* in_w, const float* weight, const float* bias, int centred, void* normed,
                                    int out_dtype, const int* rows, int n, int streams, int width, float eps, cudaStream_t stream) {
    if (n < 0 || width <= 0 || streams <= 0 || streams > MAX_STREAMS)
        return fail(MLB_UNSUPPORTED_SIZE, "streams_mix_norm: %d streams (at most %d), width %d", streams, MAX_STREAMS, width);
    if (!x || !in_w || !weight || !normed || (y && (n_y < 1 || !mix || !out_w)))
        return fail(MLB_INVALID_ARGUMENT, "streams_mix_norm: bad operands");
    if (n == 0) return MLB_OK;
    StreamParams p{x, y, n_y, y ? y_stride : 0, mix, out_w, in_w, weight, bias, centred ? 1 : 0, eps, normed, rows, streams, width};
    if (out_dtype == MLB_BF16) return launch<__nv_bfloat16>(p, n, stream);
    if (out_dtype == MLB_F32) return launch<float>(p, n, stream);
    return fail(MLB_INVALID_ARGUMENT, "streams_mix_norm: unsupported output dtype %d", out_dtype);
}

MLB_EXPORT int mlb_streams_total(const float* x, const float* y, int n_y, long long y_stride, const float* mix, const float* out_w,
                                 float* out, int n, int streams, int width, cudaStream_t stream) {
    if (n < 0 || width <= 0 || streams <= 0 || streams > MAX_STREAMS) return fail(MLB_UNSUPPORTED_SIZE, "streams_total: bad sizes");
    if (!x || !out || (y && (n_y < 1 || !mix || !out_w))) return fail(MLB_INVALID_ARGUMENT, "streams_total: bad operands");
    if (n == 0) return MLB_OK;
    StreamParams p{const_cast<float*>(x), y, n_y, y ? y_stride : 0, mix, out_w, nullptr, nullptr, nullptr, 0, 0.0f, nullptr, nullptr, streams, width};
    launch_kernel(total_kernel, (unsigned)n, THREADS, 0, stream, p, out);
    return check_launch("streams_total");
}
