// What happens to a fused projection's query, key and value heads between the projection and the
// attention, as one kernel: unit-RMS normalisation of query and key heads, the blend of the values
// with another layer's values of the same token, and the write of keys and values to their pages.
// (Further down: the same place of an attention whose queries, keys and values come from two latents.)
//
// One warp per (token, head) over the H query heads, the G key heads and the G value heads of a row
// [ ... q (H x D) ... k (G x D) ... v (G x Dv) ... ] whose three column offsets are parameters.
//   query head:  q <- q / sqrt(mean(q^2) + eps), in place            (if unit_norm)
//   key head:    k <- k / sqrt(mean(k^2) + eps), to its cache row    (if unit_norm; else copied)
//   value head:  v <- (1 - t) v + t v_other,      to its cache row    (if v_other is given; else copied)
// With q_gain / k_gain (head_dim numbers each, shared by the heads) the unit-RMS query and key heads
// are multiplied by them.  The value columns may be the key columns (v_off = k_off): keys are
// normalised on their way to the cache, never in place, so the values are the keys as projected.
// A query temperature (`every` > 0) multiplies the query heads of position p by 1 + coef * ln(floor((p + 1) / every) + 1),
// behind the norm and the gain, before they are rounded.
// The statistics and the blend are 32-bit; t is read from device memory.  Key pages are
// [page, kv head, page_tokens, D], value pages [page, kv head, page_tokens, Dv].  A token with a
// negative position (padding of a fixed-size batch) is skipped, a negative cache row is not written.
#include "common.cuh"

MG_GUARD_DECLARE(head_prepare)

namespace {

constexpr int WARPS = 4;
constexpr int MAX_PER_LANE = 8;     // head sizes up to 256

template <typename T>
__global__ void __launch_bounds__(32 * WARPS)
head_prepare_kernel(T* __restrict__ proj, int ld, int n_tokens, int n_head, int n_kv_head, int head_dim, int v_dim,
                    int q_off, int k_off, int v_off, int unit_norm, float eps, const T* __restrict__ v_other,
                    int v_other_ld, const float* __restrict__ blend, const int* __restrict__ slots,
                    const int* __restrict__ positions, T* __restrict__ k_pages, T* __restrict__ v_pages,
                    int page_tokens, int num_pages, const float* __restrict__ q_gain, const float* __restrict__ k_gain,
                    float temp_coef, double temp_every) {
    pdl_trigger();
    pdl_wait();                                            // the rows come from the projection in front
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int token = blockIdx.x;
    const int unit = blockIdx.y * WARPS + warp;
    if (unit >= n_head + 2 * n_kv_head) return;
    if (positions != nullptr && positions[token] < 0) return;
    T* row = proj + (size_t)token * ld;
    int slot = slots ? slots[token] : -1;
    if (slot >= 0 && !MG_GUARDED(head_prepare, MG_GUARD_CACHE_ROW, slot, (long long)num_pages * page_tokens)) slot = -1;
    const int page = slot >= 0 ? slot / page_tokens : 0, within = slot >= 0 ? slot - page * page_tokens : 0;

    if (unit < n_head + n_kv_head) {                       // a query or key head
        const bool is_key = unit >= n_head;
        const int h = is_key ? unit - n_head : unit;
        T* src = row + (is_key ? k_off : q_off) + (size_t)h * head_dim;
        float v[MAX_PER_LANE];
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_PER_LANE; ++i) {
            const int d = lane + 32 * i;
            v[i] = d < head_dim ? to_float(src[d]) : 0.f;
            sq = fmaf(v[i], v[i], sq);
        }
        const float r = unit_norm ? 1.0f / sqrtf(warp_sum(sq) / (float)head_dim + eps) : 1.0f;
        const float* gain = is_key ? k_gain : q_gain;
        T* dst = src;
        if (is_key) {
            if (k_pages == nullptr || slot < 0) return;
            dst = k_pages + (((size_t)page * n_kv_head + h) * page_tokens + within) * head_dim;
        } else if (!unit_norm && temp_every <= 0.0) {
            return;
        }
        // (the steps are counted in 64-bit: a position right at a step's edge is on its own side)
        const float temp = !is_key && temp_every > 0.0
                               ? 1.0f + temp_coef * logf((float)floor(((double)positions[token] + 1.0) / temp_every) + 1.0f) : 1.0f;
#pragma unroll
        for (int i = 0; i < MAX_PER_LANE; ++i) {
            const int d = lane + 32 * i;
            if (d < head_dim) dst[d] = from_float<T>((gain ? v[i] * r * gain[d] : v[i] * r) * temp);
        }
        return;
    }
    // a value head
    if (v_pages == nullptr || slot < 0) return;
    const int h = unit - n_head - n_kv_head;
    const T* src = row + v_off + (size_t)h * v_dim;
    const T* other = v_other ? v_other + (size_t)token * v_other_ld + (size_t)h * v_dim : nullptr;
    const float t = other ? blend[0] : 0.f;
    T* dst = v_pages + (((size_t)page * n_kv_head + h) * page_tokens + within) * v_dim;
    for (int d = lane; d < v_dim; d += 32) {
        float x = to_float(src[d]);
        if (other) x = (1.0f - t) * x + t * to_float(other[d]);
        dst[d] = from_float<T>(x);
    }
}

// Two latents of a token (stretches of its projected row), each divided by its root mean square, times its gain:
// blockIdx.y 0 takes the one behind the queries to a row of its own, 1 the one behind keys and values to the
// token's cache row.  V features at a time (8 where 16-byte accesses fit).
constexpr int LATENT_THREADS = 128;

template <typename T, int V>
__global__ void __launch_bounds__(LATENT_THREADS)
latent_pair_kernel(const T* __restrict__ proj, int ld, int q_off, int q_rank, const float* __restrict__ q_gain,
                   T* __restrict__ q_out, int low_off, int rank, const float* __restrict__ gain, float eps,
                   const int* __restrict__ positions, const int* __restrict__ slots, T* __restrict__ pages, int page_tokens,
                   int num_pages) {
    __shared__ float red[LATENT_THREADS / 32];
    pdl_trigger();
    pdl_wait();
    const int token = blockIdx.x, tid = threadIdx.x;
    const bool cached = blockIdx.y == 1;
    const int n = cached ? rank : q_rank;
    T* dst;
    if (cached) {
        int slot = slots[token];
        if (slot >= 0 && !MG_GUARDED(head_prepare, MG_GUARD_CACHE_ROW, slot, (long long)num_pages * page_tokens)) slot = -1;
        if (slot < 0 || positions[token] < 0) return;
        dst = pages + (size_t)slot * rank;                 // (one row a token and page slot)
    } else {
        dst = q_out + (size_t)token * q_rank;
    }
    const T* src = proj + (size_t)token * ld + (cached ? low_off : q_off);
    const float* w = cached ? gain : q_gain;
    float sq = 0.f;
    for (int i = tid * V; i < n; i += LATENT_THREADS * V) {
        __align__(16) T x[V];
        if constexpr (V > 1) {
#pragma unroll
            for (int u = 0; u < (int)(V * sizeof(T) / 16); ++u) reinterpret_cast<uint4*>(x)[u] = reinterpret_cast<const uint4*>(src + i)[u];
        } else {
            x[0] = src[i];
        }
#pragma unroll
        for (int u = 0; u < V; ++u) sq = fmaf(to_float(x[u]), to_float(x[u]), sq);
    }
    sq = warp_sum(sq);
    if ((tid & 31) == 0) red[tid >> 5] = sq;
    __syncthreads();
    const float total = (red[0] + red[1]) + (red[2] + red[3]);
    const float r = 1.0f / sqrtf(total / (float)n + eps);
    for (int i = tid * V; i < n; i += LATENT_THREADS * V) {
        __align__(16) T x[V];
        if constexpr (V > 1) {
#pragma unroll
            for (int u = 0; u < (int)(V * sizeof(T) / 16); ++u) reinterpret_cast<uint4*>(x)[u] = reinterpret_cast<const uint4*>(src + i)[u];
        } else {
            x[0] = src[i];
        }
#pragma unroll
        for (int u = 0; u < V; ++u) x[u] = from_float<T>(to_float(x[u]) * r * w[i + u]);
        if constexpr (V > 1) {
#pragma unroll
            for (int u = 0; u < (int)(V * sizeof(T) / 16); ++u) reinterpret_cast<uint4*>(dst + i)[u] = reinterpret_cast<const uint4*>(x)[u];
        } else {
            dst[i] = x[0];
        }
    }
}

}  // namespace

// proj: [n_tokens, ld] rows (bfloat16 if is_bf16 else 32-bit) with the queries' latent (q_rank numbers from q_off) and
// the one behind keys and values (rank numbers from low_off); q_gain: [q_rank], gain: [rank] 32-bit; q_out: [n_tokens,
// q_rank]; slots: [n_tokens] flat cache rows; positions: [n_tokens]; pages: [page, 1, page_tokens, rank].
MG_API int mg_latent_pair_prepare(const void* proj, int ld, int n_tokens, int q_off, int q_rank, const float* q_gain,
                                  void* q_out, int low_off, int rank, const float* gain, float eps, const int* positions,
                                  const int* slots, void* pages, int page_tokens, int num_pages, int is_bf16, void* stream) {
    if (n_tokens == 0) return MG_OK;
    MG_REQUIRE(n_tokens > 0 && q_rank > 0 && rank > 0 && page_tokens > 0 && positions && slots && pages && q_out && q_gain && gain,
               "latent_pair_prepare: bad sizes");
    MG_REQUIRE(q_off >= 0 && q_off + q_rank <= ld && low_off >= 0 && low_off + rank <= ld, "latent_pair_prepare: latents outside the rows");
    const dim3 grid(n_tokens, 2), block(LATENT_THREADS);
    const bool vec = ld % 8 == 0 && q_off % 8 == 0 && q_rank % 8 == 0 && low_off % 8 == 0 && rank % 8 == 0 &&
                     (uintptr_t)proj % 16 == 0 && (uintptr_t)q_out % 16 == 0 && (uintptr_t)pages % 16 == 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (is_bf16)
        e = mg_launch(vec ? latent_pair_kernel<bf16, 8> : latent_pair_kernel<bf16, 1>, grid, block, 0, s, true, (const bf16*)proj, ld,
                      q_off, q_rank, q_gain, (bf16*)q_out, low_off, rank, gain, eps, positions, slots, (bf16*)pages, page_tokens,
                      num_pages);
    else
        e = mg_launch(vec ? latent_pair_kernel<float, 8> : latent_pair_kernel<float, 1>, grid, block, 0, s, true, (const float*)proj,
                      ld, q_off, q_rank, q_gain, (float*)q_out, low_off, rank, gain, eps, positions, slots, (float*)pages,
                      page_tokens, num_pages);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "latent_pair_prepare: %s", cudaGetErrorString(e));
    return MG_OK;
}

// proj: [n_tokens, ld] rows of a fused projection (bfloat16 if is_bf16 else 32-bit), modified in place
// (query heads); v_other: [n_tokens, v_other_ld] rows whose first n_kv_head * v_dim columns are the
// values to blend in, blend: one 32-bit number on the device (both null: no blend); slots: [n_tokens]
// flat cache rows (null with the pages: nothing is cached); positions: [n_tokens] or null; q_gain, k_gain:
// [head_dim] 32-bit or null; temp_coef, temp_every: the query temperature (temp_every <= 0: none; it wants positions).
MG_API int mg_head_prepare(void* proj, int ld, int n_tokens, int n_head, int n_kv_head, int head_dim, int v_dim,
                           int q_off, int k_off, int v_off, int unit_norm, float eps, const void* v_other,
                           int v_other_ld, const float* blend, const int* slots, const int* positions, void* k_pages,
                           void* v_pages, int page_tokens, int num_pages, int is_bf16, const float* q_gain,
                           const float* k_gain, float temp_coef, double temp_every, void* stream) {
    if (n_tokens == 0) return MG_OK;
    MG_REQUIRE(n_tokens > 0 && n_head > 0 && n_kv_head > 0 && head_dim > 0 && v_dim > 0, "head_prepare: bad sizes");
    MG_REQUIRE(head_dim <= 32 * MAX_PER_LANE && v_dim <= 32 * MAX_PER_LANE, "head_prepare: heads of up to %d features",
               32 * MAX_PER_LANE);
    MG_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + n_head * head_dim <= ld &&
                   k_off + n_kv_head * head_dim <= ld && v_off + n_kv_head * v_dim <= ld,
               "head_prepare: heads outside the rows");
    MG_REQUIRE(temp_every <= 0.0 || positions != nullptr, "head_prepare: a query temperature wants positions");
    MG_REQUIRE((q_gain == nullptr && k_gain == nullptr) || unit_norm, "head_prepare: gains without the unit norm");
    MG_REQUIRE((v_other == nullptr) == (blend == nullptr), "head_prepare: a blend wants both the other values and its weight");
    MG_REQUIRE(v_other == nullptr || v_other_ld >= n_kv_head * v_dim, "head_prepare: the other values' rows are too short");
    MG_REQUIRE((k_pages == nullptr) == (v_pages == nullptr) && (k_pages == nullptr || (slots && page_tokens > 0)),
               "head_prepare: pages without cache rows");
    const dim3 grid(n_tokens, ceil_div(n_head + 2 * n_kv_head, WARPS)), block(32 * WARPS);
    MG_REQUIRE(grid.y <= 65535, "head_prepare: too many heads");
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (is_bf16)
        e = mg_launch(head_prepare_kernel<bf16>, grid, block, 0, s, true, (bf16*)proj, ld, n_tokens, n_head, n_kv_head,
                      head_dim, v_dim, q_off, k_off, v_off, unit_norm, eps, (const bf16*)v_other, v_other_ld, blend, slots,
                      positions, (bf16*)k_pages, (bf16*)v_pages, page_tokens, num_pages, q_gain, k_gain, temp_coef, temp_every);
    else
        e = mg_launch(head_prepare_kernel<float>, grid, block, 0, s, true, (float*)proj, ld, n_tokens, n_head, n_kv_head,
                      head_dim, v_dim, q_off, k_off, v_off, unit_norm, eps, (const float*)v_other, v_other_ld, blend, slots,
                      positions, (float*)k_pages, (float*)v_pages, page_tokens, num_pages, q_gain, k_gain, temp_coef, temp_every);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "head_prepare: %s", cudaGetErrorString(e));
    return MG_OK;
}
