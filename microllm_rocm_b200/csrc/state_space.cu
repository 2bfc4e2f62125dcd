// What surrounds a selective state-space recurrence (one decay and one step size per token and head; the recurrence itself is
// mlb_head_scan in delta_rule.cu, the convolution in front of it mlb_short_conv).  fp32 arithmetic throughout; only what a
// product reads next is stored in the compute dtype.
//
//   mlb_ssm_steps          dt[t, h] = softplus(proj[t, dt_col + h] + dt_bias[h]) and decay[t, h] = exp(-exp(A_log[h]) dt[t, h]), out
//                          of a projection's fp32 output (K-split partial results summed in split order).  In the same launch,
//                          optionally, the convolution's state moves on: the last taps - 1 inputs of every sequence of the step
//                          (it must run behind the convolution, which reads the old state).
//   mlb_gated_group_norm   y = (o + D_h x) * silu(z), divided by the root mean square of each of `groups` equal parts of the row
//                          (the gate comes first), times a weight of the row's length.
#include "common.cuh"

using namespace mlb;

MLB_DEFINE_LAST_ERROR()

namespace {

constexpr int MAX_HIST = 16;

struct Columns {               // a block of columns of fp32 rows, possibly K-split partial results
    const float* base; long long ld; int n_partials; long long partial_stride;
    __device__ __forceinline__ float at(long long row, int col) const {
        const float* p = base + row * ld + col;
        float v = p[0];
        for (int k = 1; k < n_partials; ++k) v += p[(size_t)k * partial_stride];
        return v;
    }
    __device__ __forceinline__ float4 at4(long long row, int col) const {      // four columns, 16-byte aligned
        const float* p = base + row * ld + col;
        float4 v = *reinterpret_cast<const float4*>(p);
        for (int k = 1; k < n_partials; ++k) {
            const float4 w = *reinterpret_cast<const float4*>(p + (size_t)k * partial_stride);
            v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
        }
        return v;
    }
    __host__ bool fours(int col) const {
        return ((uintptr_t)base % 16 == 0) && ld % 4 == 0 && col % 4 == 0 && (n_partials <= 1 || partial_stride % 4 == 0);
    }
};

__device__ __forceinline__ float softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float silu(float v) { return v / (1.0f + expf(-v)); }

// ------------------------------------------------------------------------------ step sizes, decays, the convolution's state
struct StepsParams {
    Columns proj; int dt_col;
    const float* dt_bias; const float* a_log;      // [H]
    float* dt; float* decay;                       // [T, H]
    int T, H;
    int conv_col, channels, hist;                  // hist 0: no state to move
    float* conv_state;                             // [slots + 1, hist, channels], oldest first
    const int* slots; int num_slots; const int* seq_starts; int A;
};

__global__ void ssm_steps_kernel(StepsParams p, long long step_threads) {
    pdl_prologue();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < step_threads) {                        // (a multiple of the block's size: no block does both)
        if (i >= (long long)p.T * p.H) return;
        const long long t = i / p.H;
        const int h = (int)(i % p.H);
        const float dt = softplus(p.proj.at(t, p.dt_col + h) + p.dt_bias[h]);
        p.dt[i] = dt;
        p.decay[i] = expf(-expf(p.a_log[h]) * dt);
        return;
    }
    i -= step_threads;
    if (i >= (long long)p.A * p.channels) return;
    const int a = (int)(i / p.channels), c = (int)(i % p.channels);
    const int start = p.seq_starts[a], n = p.seq_starts[a + 1] - start;
    const int slot = p.slots[a];
    if (slot < 0 || slot >= p.num_slots || n <= 0) return;
    float* st = p.conv_state + (size_t)slot * p.hist * p.channels + c;
    float keep[MAX_HIST];
#pragma unroll
    for (int m = 0; m < MAX_HIST; ++m) {
        if (m >= p.hist) break;
        const int src = n - p.hist + m;
        keep[m] = src >= 0 ? p.proj.at((long long)start + src, p.conv_col + c) : st[(size_t)(m + n) * p.channels];
    }
#pragma unroll
    for (int m = 0; m < MAX_HIST; ++m) {
        if (m >= p.hist) break;
        st[(size_t)m * p.channels] = keep[m];
    }
}

// ------------------------------------------------------------------------------ skip, gate and norm of the result
struct GroupNormParams {
    const float* o;                          // [T, H * DV]
    const float* x; long long ld_x;          // [T, H * DV] rows ld_x apart: what entered the recurrence
    const float* d;                          // [H]
    Columns z; int z_col;
    const float* weight;                     // [H * DV]
    void* out;                               // [T, H * DV]
    int T, DV, width, groups; float eps;
};

// THREADS threads share one (token, group): a warp of a block of four, or a whole block of 256.  Up to PER elements (X4: groups
// of four) a thread stay in registers; longer parts are read a second time.
template <typename OutT, int THREADS, bool X4>
__global__ void __launch_bounds__(THREADS == 32 ? 128 : THREADS) gated_group_norm_kernel(GroupNormParams p) {
    constexpr int PER = X4 ? 4 : 16, STEP = X4 ? 4 : 1;
    pdl_prologue();
    __shared__ float scratch[32];
    const long long item = THREADS == 32 ? (long long)blockIdx.x * 4 + (threadIdx.x >> 5) : blockIdx.x;
    if (item >= (long long)p.T * p.groups) return;               // (a whole warp, or never)
    const long long t = item / p.groups;
    const int group = (int)(item % p.groups), size = p.width / p.groups, c0 = group * size;
    const int me = THREADS == 32 ? (threadIdx.x & 31) : threadIdx.x;
    const float* const o = p.o + (size_t)t * p.width;
    const float* const x = p.x + (size_t)t * p.ld_x;
    auto one = [&](int c) { return fmaf(p.d[c / p.DV], x[c], o[c]) * silu(p.z.at(t, p.z_col + c)); };
    auto four = [&](int c) {                 // four neighbours belong to one head
        const float4 a = *reinterpret_cast<const float4*>(o + c), b = *reinterpret_cast<const float4*>(x + c), g = p.z.at4(t, p.z_col + c);
        const float d = p.d[c / p.DV];
        return make_float4(fmaf(d, b.x, a.x) * silu(g.x), fmaf(d, b.y, a.y) * silu(g.y), fmaf(d, b.z, a.z) * silu(g.z), fmaf(d, b.w, a.w) * silu(g.w));
    };
    float y[PER * STEP];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int c = (me + i * THREADS) * STEP;
        if (X4) {
            const float4 v = c < size ? four(c0 + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            y[i * STEP] = v.x; y[i * STEP + STEP / 4] = v.y; y[i * STEP + STEP / 2] = v.z; y[i * STEP + STEP - 1] = v.w;
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
        } else {
            y[i] = c < size ? one(c0 + c) : 0.0f;
            ss = fmaf(y[i], y[i], ss);
        }
    }
    for (int c = me + PER * STEP * THREADS; c < size; c += THREADS) { const float v = one(c0 + c); ss = fmaf(v, v, ss); }
    ss = THREADS == 32 ? warp_sum(ss) : block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)size + p.eps);
    OutT* const out = (OutT*)p.out + (size_t)t * p.width + c0;
    const float* const w = p.weight + c0;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int c = (me + i * THREADS) * STEP;
        if (c >= size) continue;
        if (X4) {
            const float4 k = *reinterpret_cast<const float4*>(w + c);
            const float r[4] = {y[i * STEP] * inv * k.x, y[i * STEP + STEP / 4] * inv * k.y, y[i * STEP + STEP / 2] * inv * k.z,
                                y[i * STEP + STEP - 1] * inv * k.w};
            if constexpr (sizeof(OutT) == 2) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
                uint2 raw = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
                *reinterpret_cast<uint2*>(out + c) = raw;
            } else {
                *reinterpret_cast<float4*>(out + c) = make_float4(r[0], r[1], r[2], r[3]);
            }
        } else {
            out[c] = from_f32<OutT>(y[i] * inv * w[c]);
        }
    }
    for (int c = me + PER * STEP * THREADS; c < size; c += THREADS) out[c] = from_f32<OutT>(one(c0 + c) * inv * w[c]);
}

template <typename OutT>
void launch_group_norm(const GroupNormParams& p, bool x4, cudaStream_t stream) {
    const long long items = (long long)p.T * p.groups;
    const int size = p.width / p.groups;
    if (size <= 512) {
        const unsigned blocks = (unsigned)((items + 3) / 4);
        if (x4) launch_kernel(gated_group_norm_kernel<OutT, 32, true>, blocks, 128, 0, stream, p);
        else launch_kernel(gated_group_norm_kernel<OutT, 32, false>, blocks, 128, 0, stream, p);
        return;
    }
    if (x4) launch_kernel(gated_group_norm_kernel<OutT, 256, true>, (unsigned)items, 256, 0, stream, p);
    else launch_kernel(gated_group_norm_kernel<OutT, 256, false>, (unsigned)items, 256, 0, stream, p);
}

}  // namespace

MLB_EXPORT int mlb_ssm_steps(const float* proj, long long ld, int n_partials, long long partial_stride, int dt_col, const float* dt_bias,
                             const float* a_log, float* dt, float* decay, int T, int H, int conv_col, int channels, int hist,
                             float* conv_state, const int* slots, int num_slots, const int* seq_starts, int A, cudaStream_t stream) {
    if (T < 0 || H <= 0 || A < 0 || channels < 0 || hist < 0 || hist > MAX_HIST || !proj || !dt_bias || !a_log || !dt || !decay)
        return fail(MLB_INVALID_ARGUMENT, "ssm_steps: bad operands (a history of at most %d)", MAX_HIST);
    if (hist > 0 && (!conv_state || !slots || !seq_starts || num_slots <= 0)) return fail(MLB_INVALID_ARGUMENT, "ssm_steps: a state to move needs its slots");
    if (T == 0) return MLB_OK;
    StepsParams p{Columns{proj, ld, n_partials < 1 ? 1 : n_partials, partial_stride}, dt_col, dt_bias, a_log, dt, decay, T, H,
                  conv_col, channels, hist, conv_state, slots, num_slots, seq_starts, A};
    const long long step_threads = ((long long)T * H + 127) / 128 * 128;
    const long long all = step_threads + (hist > 0 ? (long long)A * channels : 0);
    launch_kernel(ssm_steps_kernel, (unsigned)((all + 127) / 128), 128, 0, stream, p, step_threads);
    return check_launch("ssm_steps");
}

MLB_EXPORT int mlb_gated_group_norm(const float* o, const float* x, long long ld_x, const float* d, const float* z, long long ld_z,
                                    int z_partials, long long z_partial_stride, int z_col, const float* weight, void* out, int out_dtype,
                                    int T, int H, int DV, int groups, float eps, cudaStream_t stream) {
    const int width = H * DV;
    if (T < 0 || H <= 0 || DV <= 0 || groups <= 0 || width % groups || !o || !x || !d || !z || !weight || !out || ld_x < width)
        return fail(MLB_INVALID_ARGUMENT, "gated_group_norm: %d groups of %d columns", groups, width);
    if (T == 0) return MLB_OK;
    GroupNormParams p{o, x, ld_x, d, Columns{z, ld_z, z_partials < 1 ? 1 : z_partials, z_partial_stride}, z_col, weight, out, T, DV, width, groups, eps};
    const bool x4 = (width / groups) % 4 == 0 && DV % 4 == 0 && ld_x % 4 == 0 && p.z.fours(z_col) &&
                    ((uintptr_t)o | (uintptr_t)x | (uintptr_t)weight | (uintptr_t)out) % 16 == 0;
    if (out_dtype == MLB_BF16) launch_group_norm<__nv_bfloat16>(p, x4, stream);
    else if (out_dtype == MLB_F32) launch_group_norm<float>(p, x4, stream);
    else return fail(MLB_INVALID_ARGUMENT, "gated_group_norm: unknown output dtype %d", out_dtype);
    return check_launch("gated_group_norm");
}
