// Attention over a compressed key/value cache ("latent attention").
//
// Per token the cache holds ONE row for all heads: c[R] (the normalised latent from which every head's key and
// value would be expanded, k_h = Wuk_h c, v_h = Wuv_h c) followed by kr[Dr] (a rotated key part that all heads
// share).  The expansion is never materialised: with a[h] = Wuk_h^T q_h (computed by a product per head before this
// kernel) the score of head h against key j is
//
//     s = (a[h] . c_j + qr[h] . kr_j) * scale
//
// and the head's output in latent space is sum_j p_j c_j, which a second product per head turns into Wuv_h (sum_j p_j c_j).
// So every head attends to the same rows: Dk = R + Dr wide for the score, the first R of them again as the value.
//
//   latent_prepare   from the fused projection output [T, ld] fp32 (or its split partial sums):
//                      columns q_col..   : H heads of (dim plain, Dr rotated) query elements
//                      columns kv_col..  : R latent elements, then Dr shared rotated-key elements
//                      columns gate_col..: gate_width pre-activations of an output gate (optional)
//                    -> q_plain[T, H*dim]           the plain query parts, input of the product with Wuk
//                       q_full[T, H*(R+Dr)]         only its last Dr columns per head: the rotated query parts
//                       pages[page, slot, 0:R]      c = rms(latent) * norm_weight;  [R:R+Dr] = rotated kr
//                       gate_out[T, gate_width]     sigmoid of the pre-activations, fp32
//                    rotation: element i of the first rot_dims is paired with i + rot_dims/2 (or, interleaved, 2i with 2i + 1),
//                    angle = pos * inv_freq[pair], cosines and sines times `magnitude`
//   latent_compress  for queries that come out of a latent of their own (a product follows before latent_prepare can split
//                    them): the cache row as above, and c_q[T, RQ] = rms(columns cq_col..) * its weight in the compute dtype
//   latent_attention_plain   one warp per (token, head); keys in tiles of 32 at absolute multiples of 32, running
//                    maximum and sum in fp32; a learned per-head sink enters the denominator once, unscaled, with
//                    no value.  Bit-stable under any cutting of the tokens into steps.
#include "common.cuh"

using namespace mlb;

MLB_DEFINE_LAST_ERROR()

namespace {

struct PrepareParams {
    const float* proj; long long ld; int n_partials; long long partial_stride;
    long long q_col, kv_col, gate_col;
    const float* norm_weight; float eps;
    const int* positions; const int* token_seq; const int* block_table; int max_blocks;
    const float* inv_freq; int rot_dims; int interleaved; float magnitude;
    void* q_plain; void* q_full; void* pages; float* gate_out;
    int num_pages, page_size, tokens, heads, dim, rot_dim, rank, gate_width;
    int* error_flag;
    // latent_compress only
    long long cq_col; int cq_rank; const float* cq_weight; void* cq_out;
};

// where the partner of element i of a rotated part sits, which pair they are, and whether i is the pair's first element
struct Pair { int other, index; bool first; };
__device__ __forceinline__ Pair pair_of(int i, int half, int interleaved) {
    if (interleaved) return Pair{i ^ 1, i >> 1, (i & 1) == 0};
    return i < half ? Pair{i + half, i, true} : Pair{i - half, i - half, false};
}

__device__ __forceinline__ float turned(float v, float other, bool first, float angle, float magnitude) {
    const float cs = cosf(angle) * magnitude, sn = sinf(angle) * magnitude;
    return first ? v * cs - other * sn : v * cs + other * sn;
}

__device__ __forceinline__ float proj_at(const PrepareParams& p, size_t row_base, long long col) {
    float v = p.proj[row_base + col];
    for (int k = 1; k < p.n_partials; ++k) v += p.proj[(size_t)k * p.partial_stride + row_base + col];
    return v;
}

constexpr int SLICE = 1024;        // query and gate columns per block

// A block's share of a row's norm: up to ROW_PER elements a thread stay in registers, fetched side by side (the partial results of
// all of them a step of the sum at a time), so that a decode step's few rows pay one trip to memory; longer rows are read twice.
constexpr int ROW_PER = 4;
template <typename OutT>
__device__ __forceinline__ void normed_row(const PrepareParams& p, size_t row, long long col, int n, const float* __restrict__ weight,
                                           const float (&w)[ROW_PER], const float (&v)[ROW_PER], float* scratch, OutT* out) {
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < ROW_PER; ++i) ss = fmaf(v[i], v[i], ss);                   // (zero beyond the row)
    for (int c = threadIdx.x + ROW_PER * blockDim.x; c < n; c += blockDim.x) { const float u = proj_at(p, row, col + c); ss = fmaf(u, u, ss); }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + p.eps);
    if (!out) return;
#pragma unroll
    for (int i = 0; i < ROW_PER; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n) out[c] = from_f32<OutT>(v[i] * inv * w[i]);
    }
    for (int c = threadIdx.x + ROW_PER * blockDim.x; c < n; c += blockDim.x) out[c] = from_f32<OutT>(proj_at(p, row, col + c) * inv * weight[c]);
}
__device__ __forceinline__ void fetch_row(const PrepareParams& p, size_t row, long long col, int n, float (&v)[ROW_PER]) {
#pragma unroll
    for (int i = 0; i < ROW_PER; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        v[i] = c < n ? p.proj[row + col + c] : 0.0f;
    }
#pragma unroll 4
    for (int k = 1; k < p.n_partials; ++k) {
        const float* const at = p.proj + (size_t)k * p.partial_stride + row + col;
#pragma unroll
        for (int i = 0; i < ROW_PER; ++i) {
            const int c = threadIdx.x + i * blockDim.x;
            if (c < n) v[i] += at[c];
        }
    }
}
__device__ __forceinline__ void fetch_weight(const float* __restrict__ weight, int n, float (&w)[ROW_PER]) {
#pragma unroll
    for (int i = 0; i < ROW_PER; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        w[i] = weight && c < n ? weight[c] : 0.0f;
    }
}

// The token's cache row: the normalised latent, and behind it the shared key part with its rotation.  `w`: the norm's weights of
// this thread (fetched before the wait for the predecessor).
template <typename KVT>
__device__ __forceinline__ void store_cache_row(const PrepareParams& p, int t, size_t row, int pos, const float (&w)[ROW_PER], float* scratch) {
    if (!p.pages) return;
    const int half = p.rot_dims / 2;
    const int Dk = p.rank + p.rot_dim;
    float v[ROW_PER];
    fetch_row(p, row, p.kv_col, p.rank, v);
    KVT* cache_row = nullptr;
    const int block = pos / p.page_size;
    const int page = block < p.max_blocks ? p.block_table[(size_t)p.token_seq[t] * p.max_blocks + block] : -1;
    if (page < 0 || page >= p.num_pages) {
        if (threadIdx.x == 0 && p.error_flag) atomicExch(p.error_flag, 1);
    } else {
        cache_row = (KVT*)p.pages + ((size_t)page * p.page_size + pos % p.page_size) * Dk;
        // the shared key part: its first rot_dims elements turned in pairs, the rest passed on
        for (int i = threadIdx.x; i < p.rot_dim; i += blockDim.x) {
            float out = proj_at(p, row, p.kv_col + p.rank + i);
            if (i < p.rot_dims) {
                const Pair pr = pair_of(i, half, p.interleaved);
                out = turned(out, proj_at(p, row, p.kv_col + p.rank + pr.other), pr.first, (float)pos * p.inv_freq[pr.index], p.magnitude);
            }
            cache_row[p.rank + i] = from_f32<KVT>(out);
        }
    }
    normed_row(p, row, p.kv_col, p.rank, p.norm_weight, w, v, scratch, cache_row);
}

template <typename QT, typename KVT>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(PrepareParams p) {
    pdl_launch_dependents();
    float w[ROW_PER];
    fetch_weight(p.pages && blockIdx.y == 0 ? p.norm_weight : nullptr, p.rank, w);
    pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const size_t row = (size_t)t * p.ld;
    const int pos = p.positions[t];
    const int half = p.rot_dims / 2;
    const int Dk = p.rank + p.rot_dim;

    // blockIdx.y == 0: the token's cache row; blockIdx.y >= 1: a slice of SLICE query and gate columns
    if (blockIdx.y > 0) {
        const int per_head = p.dim + p.rot_dim;
        const int q_cols = p.heads * per_head;
        const int lo = (blockIdx.y - 1) * SLICE, hi = min(lo + SLICE, q_cols + (p.gate_out ? p.gate_width : 0));
        for (int e = lo + threadIdx.x; e < hi; e += blockDim.x) {
            if (e >= q_cols) {                                   // the gate's sigmoid
                const int c = e - q_cols;
                const float z = proj_at(p, row, p.gate_col + c);
                p.gate_out[(size_t)t * p.gate_width + c] = 1.0f / (1.0f + expf(-z));
                continue;
            }
            // queries: plain parts to q_plain, rotated parts into the tail of each head's row of q_full
            const int h = e / per_head, i = e % per_head;
            const float v = proj_at(p, row, p.q_col + e);
            if (i < p.dim) {
                ((QT*)p.q_plain)[((size_t)t * p.heads + h) * p.dim + i] = from_f32<QT>(v);
                continue;
            }
            const int r = i - p.dim;
            float out = v;
            if (r < p.rot_dims) {
                const Pair pr = pair_of(r, half, p.interleaved);
                const float other = proj_at(p, row, p.q_col + (long long)h * per_head + p.dim + pr.other);
                out = turned(v, other, pr.first, (float)pos * p.inv_freq[pr.index], p.magnitude);
            }
            ((QT*)p.q_full)[((size_t)t * p.heads + h) * Dk + p.rank + r] = from_f32<QT>(out);
        }
        return;
    }
    store_cache_row<KVT>(p, t, row, pos, w, scratch);
}

// One block per token and part: blockIdx.y 0 the cache row, 1 the queries' latent.
constexpr int COMPRESS_THREADS = 128;
template <typename QT, typename KVT>
__global__ void __launch_bounds__(COMPRESS_THREADS)
latent_compress_kernel(PrepareParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const size_t row = (size_t)t * p.ld;
    float w[ROW_PER];
    fetch_weight(blockIdx.y == 0 ? p.norm_weight : p.cq_weight, blockIdx.y == 0 ? p.rank : p.cq_rank, w);
    pdl_wait();
    if (blockIdx.y == 0) {
        store_cache_row<KVT>(p, t, row, p.positions[t], w, scratch);
        return;
    }
    float v[ROW_PER];
    fetch_row(p, row, p.cq_col, p.cq_rank, v);
    normed_row(p, row, p.cq_col, p.cq_rank, p.cq_weight, w, v, scratch, (QT*)p.cq_out + (size_t)t * p.cq_rank);
}

constexpr int WARPS = 4;
constexpr int MAX_DK = 640;
constexpr int MAX_R = 512;

struct AttnParams {
    const void* q;           // [T, H*(R+Dr)]
    const void* pages;       // [num_pages, page_size, R+Dr]
    void* out;               // [T, H*R]
    const float* sink;       // [H] or null
    const int* positions; const int* token_seq; const int* block_table;
    int max_blocks, num_pages, page_size, tokens, heads, rank, rot_dim, window;
    float scale;
    int* error_flag;
};

template <typename QT, typename KVT, typename OutT>
__global__ void __launch_bounds__(WARPS * 32)
latent_attention_plain_kernel(AttnParams p) {
    pdl_prologue();
    __shared__ float q_s[WARPS][MAX_DK];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    if (item >= (long long)p.tokens * p.heads) return;
    const int t = (int)(item / p.heads), h = (int)(item % p.heads);
    const int R = p.rank, Dk = p.rank + p.rot_dim;
    const int pos = p.positions[t];
    const int seq = p.token_seq[t];
    const int lo = (p.window > 0 && pos - p.window + 1 > 0) ? pos - p.window + 1 : 0;
    const QT* qrow = (const QT*)p.q + ((size_t)t * p.heads + h) * Dk;
    for (int c = lane; c < Dk; c += 32) q_s[warp][c] = to_f32(qrow[c]);
    __syncwarp();

    constexpr int PER_LANE = MAX_R / 32;
    float acc[PER_LANE];
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) acc[i] = 0.0f;
    // the sink is one more term of the denominator: exp(sink) with no key and no value
    float m = p.sink ? p.sink[h] : -INFINITY;
    float l = p.sink ? 1.0f : 0.0f;
    const int* table = p.block_table + (size_t)seq * p.max_blocks;

    for (int base = (lo / 32) * 32; base <= pos; base += 32) {
        const int kp = base + lane;
        bool valid = kp >= lo && kp <= pos;
        long long k_off = -1;
        if (valid) {
            const int block = kp / p.page_size;
            const int page = block < p.max_blocks ? table[block] : -1;
            if (page < 0 || page >= p.num_pages) {
                if (p.error_flag) atomicExch(p.error_flag, 2);
                valid = false;
            } else {
                k_off = (long long)(((size_t)page * p.page_size + kp % p.page_size) * Dk);
            }
        }
        float s = -INFINITY;
        if (valid) {
            const KVT* krow = (const KVT*)p.pages + k_off;
            float dot = 0.0f;
            for (int c = 0; c < Dk; ++c) dot = fmaf(q_s[warp][c], to_f32(krow[c]), dot);
            s = dot * p.scale;
        }
        const float m_new = fmaxf(m, warp_max(s));
        if (m_new == -INFINITY) continue;
        const float prob = valid ? expf(s - m_new) : 0.0f;
        const float corr = (m == -INFINITY) ? 0.0f : expf(m - m_new);
        l = l * corr + warp_sum(prob);
        m = m_new;
#pragma unroll
        for (int i = 0; i < PER_LANE; ++i) acc[i] *= corr;
        const unsigned valid_mask = __ballot_sync(0xffffffffu, valid);
        for (int j = 0; j < 32; ++j) {
            const float pj = __shfl_sync(0xffffffffu, prob, j);
            const long long off_j = __shfl_sync(0xffffffffu, k_off, j);
            if (!((valid_mask >> j) & 1u)) continue;
            const KVT* vrow = (const KVT*)p.pages + off_j;
#pragma unroll
            for (int i = 0; i < PER_LANE; ++i) {
                const int c = lane + 32 * i;
                if (c < R) acc[i] = fmaf(pj, to_f32(vrow[c]), acc[i]);
            }
        }
    }
    OutT* orow = (OutT*)p.out + ((size_t)t * p.heads + h) * R;
    const float inv = l > 0.0f ? 1.0f / l : 0.0f;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
        const int c = lane + 32 * i;
        if (c < R) orow[c] = from_f32<OutT>(acc[i] * inv);
    }
}

}  // namespace

MLB_EXPORT int mlb_latent_prepare(const float* proj, long long ld, int n_partials, long long partial_stride, long long q_col,
                                  long long kv_col, long long gate_col, const float* norm_weight, float eps,
                                  const int* positions, const int* token_seq, const int* block_table, int max_blocks,
                                  const float* inv_freq, int rot_dims, int interleaved, float magnitude, void* q_plain, void* q_full, int q_dtype, void* pages,
                                  int kv_dtype, float* gate_out, int num_pages, int page_size, int tokens, int heads, int dim,
                                  int rot_dim, int rank, int gate_width, int* error_flag, cudaStream_t stream) {
    if (tokens < 0 || heads <= 0 || dim <= 0 || rot_dim < 0 || rank <= 0 || n_partials < 1 || !(eps > 0.0f))
        return fail(MLB_INVALID_ARGUMENT, "latent_prepare: bad sizes");
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > rot_dim) return fail(MLB_INVALID_ARGUMENT, "latent_prepare: rot_dims %d must be even and at most %d", rot_dims, rot_dim);
    if (pages && (page_size <= 0 || num_pages <= 0 || max_blocks <= 0)) return fail(MLB_INVALID_ARGUMENT, "latent_prepare: bad cache geometry");
    if (tokens == 0) return MLB_OK;
    PrepareParams p{proj, ld, n_partials, partial_stride, q_col, kv_col, gate_col, norm_weight, eps, positions, token_seq,
                    block_table, max_blocks, inv_freq, rot_dims, interleaved, magnitude, q_plain, q_full, pages, gate_out, num_pages, page_size,
                    tokens, heads, dim, rot_dim, rank, gate_width, error_flag, 0, 0, nullptr, nullptr};
    const int columns = heads * (dim + rot_dim) + (gate_out ? gate_width : 0);
    const dim3 grid(tokens, 1 + (columns + SLICE - 1) / SLICE);
    if (q_dtype == MLB_F32 && (kv_dtype == MLB_F32 || !pages))
        launch_kernel(latent_prepare_kernel<float, float>, grid, 256, 0, stream, p);
    else if (q_dtype == MLB_BF16 && (kv_dtype == MLB_BF16 || !pages))
        launch_kernel(latent_prepare_kernel<__nv_bfloat16, __nv_bfloat16>, grid, 256, 0, stream, p);
    else
        return fail(MLB_INVALID_ARGUMENT, "latent_prepare: unsupported dtypes %d / %d", q_dtype, kv_dtype);
    return check_launch("latent_prepare");
}

// the cache row of every token (pages may be null: none is stored) and c_q [tokens, cq_rank] out of one projection
MLB_EXPORT int mlb_latent_compress(const float* proj, long long ld, int n_partials, long long partial_stride, long long cq_col, int cq_rank,
                                   const float* cq_weight, void* cq_out, int q_dtype, long long kv_col, const float* norm_weight, float eps,
                                   const int* positions, const int* token_seq, const int* block_table, int max_blocks,
                                   const float* inv_freq, int rot_dims, int interleaved, float magnitude, void* pages, int kv_dtype,
                                   int num_pages, int page_size, int tokens, int rot_dim, int rank, int* error_flag, cudaStream_t stream) {
    if (tokens < 0 || cq_rank <= 0 || rot_dim < 0 || rank <= 0 || n_partials < 1 || !(eps > 0.0f) || !proj || !cq_weight || !cq_out || !norm_weight)
        return fail(MLB_INVALID_ARGUMENT, "latent_compress: bad operands");
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > rot_dim) return fail(MLB_INVALID_ARGUMENT, "latent_compress: rot_dims %d must be even and at most %d", rot_dims, rot_dim);
    if (pages && (page_size <= 0 || num_pages <= 0 || max_blocks <= 0)) return fail(MLB_INVALID_ARGUMENT, "latent_compress: bad cache geometry");
    if (tokens == 0) return MLB_OK;
    PrepareParams p{};
    p.proj = proj; p.ld = ld; p.n_partials = n_partials; p.partial_stride = partial_stride; p.kv_col = kv_col; p.norm_weight = norm_weight; p.eps = eps;
    p.positions = positions; p.token_seq = token_seq; p.block_table = block_table; p.max_blocks = max_blocks; p.inv_freq = inv_freq;
    p.rot_dims = rot_dims; p.interleaved = interleaved; p.magnitude = magnitude; p.pages = pages; p.num_pages = num_pages; p.page_size = page_size;
    p.tokens = tokens; p.rot_dim = rot_dim; p.rank = rank; p.error_flag = error_flag;
    p.cq_col = cq_col; p.cq_rank = cq_rank; p.cq_weight = cq_weight; p.cq_out = cq_out;
    const dim3 grid(tokens, 2);
    if (q_dtype == MLB_F32 && (kv_dtype == MLB_F32 || !pages)) launch_kernel(latent_compress_kernel<float, float>, grid, COMPRESS_THREADS, 0, stream, p);
    else if (q_dtype == MLB_BF16 && (kv_dtype == MLB_BF16 || !pages))
        launch_kernel(latent_compress_kernel<__nv_bfloat16, __nv_bfloat16>, grid, COMPRESS_THREADS, 0, stream, p);
    else return fail(MLB_INVALID_ARGUMENT, "latent_compress: unsupported dtypes %d / %d", q_dtype, kv_dtype);
    return check_launch("latent_compress");
}

MLB_EXPORT int mlb_latent_attention_plain(const void* q, int q_dtype, const void* pages, int kv_dtype, void* out, int out_dtype,
                                          const float* sink, const int* positions, const int* token_seq,
                                          const int* block_table, int max_blocks, int num_pages, int page_size, int tokens,
                                          int heads, int rank, int rot_dim, int window, float scale, int* error_flag,
                                          cudaStream_t stream) {
    if (tokens < 0 || heads <= 0 || rank <= 0 || rot_dim < 0) return fail(MLB_INVALID_ARGUMENT, "latent_attention_plain: bad sizes");
    if (rank > MAX_R || rank + rot_dim > MAX_DK)
        return fail(MLB_UNSUPPORTED_SIZE, "latent_attention_plain: latent %d + rotated %d exceed %d / %d", rank, rot_dim, MAX_R, MAX_DK);
    if (page_size <= 0 || num_pages <= 0 || max_blocks <= 0 || window < 0) return fail(MLB_INVALID_ARGUMENT, "latent_attention_plain: bad cache geometry");
    if (tokens == 0) return MLB_OK;
    AttnParams p{q, pages, out, sink, positions, token_seq, block_table, max_blocks, num_pages, page_size, tokens, heads, rank,
                 rot_dim, window, scale, error_flag};
    const long long items = (long long)tokens * heads;
    const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
    if (q_dtype == MLB_F32 && kv_dtype == MLB_F32 && out_dtype == MLB_F32)
        launch_kernel(latent_attention_plain_kernel<float, float, float>, blocks, WARPS * 32, 0, stream, p);
    else if (q_dtype == MLB_BF16 && kv_dtype == MLB_BF16 && out_dtype == MLB_BF16)
        launch_kernel(latent_attention_plain_kernel<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>, blocks, WARPS * 32, 0, stream, p);
    else
        return fail(MLB_INVALID_ARGUMENT, "latent_attention_plain: unsupported dtypes %d/%d/%d", q_dtype, kv_dtype, out_dtype);
    return check_launch("latent_attention_plain");
}
