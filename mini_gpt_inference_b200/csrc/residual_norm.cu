// What a layer with a norm on both sides of each sublayer, a loop over layers with an additive re-entry, and a
// per-layer token input add to the 32-bit residual stream; all sums and statistics 32-bit.
//
// norm_add:     x += scale * (y / sqrt(mean(y^2) + eps)) * (offset + w),  y = sa * a [+ sb * b]  (the sublayer's output a,
//               or the weighted sum of two sublayers that ran side by side), or the sum of the rows that a token's
//               entries point to (experts that wrote their results apart); with `center` the mean of y is taken off
//               first (a layer norm).  With `clear` the inputs are left as zeros: the buffer a sublayer added its output
//               into serves the next sublayer as it is.  Optionally the new x is also written in bfloat16 (what a
//               sublayer that reads the stream itself wants next), or an RMS norm of it, x / sqrt(mean(x^2) + eps2) *
//               (offset2 + w2), in bfloat16 or 32-bit (what a sublayer with a norm in front of it wants next)
// add_rows:     x += [e] + v    (e: rows like x, or none; v: one row for all tokens)
// scaled_sum:   x += sa * a + sb * b   (with `clear`, a and b are left as zeros)
// softcap:      x <- cap * tanh(x / cap)
// token_gate:   out[t, j] = gelu_tanh(g[t, j]) * table[token_t, off + j]   (a slice of a second embedding table as a
//               gate's other factor; tokens that the step before sampled are taken from its ids, as in the embedding)
// cast_rows:    32-bit rows in the compute type, optionally through tanh
#include <math.h>

#include "common.cuh"

MG_GUARD_DECLARE(residual_norm)

namespace {

constexpr int NORM_WARPS = 4;
constexpr int ROW_THREADS = 256;   // threads of the CTA that owns a row in the vector form
constexpr int MAX_ROW_VECS = 8;    // most float4 a thread holds: rows of up to 256 * 8 * 4 = 8,192 numbers

// What the norm behind a sublayer reads: y = sa * a [+ sb * b], or, with `entry_slot`, the sum over a row's `top` entries
// of the rows of `a` that they point to (entries below zero: none), in entry order.
struct NormInput {
    float* a;
    float sa;
    float* b;
    float sb;
    const int* entry_slot;         // [rows, top] or null
    int top, n_slots;
};

struct NormOutput {
    float* x;                      // the stream, in place
    const float* w;
    float eps, offset, scale;      // x += scale * norm(y) * (offset + w)
    int center;                    // take the row's mean off first (a layer norm)
    int clear;                     // leave a and b as zeros
    bf16* rows;                    // the new stream (with w2: its norm) in bfloat16 as well, or null
    float* rows32;                 // with w2: its norm in 32-bit, or null
    const float* w2;               // the weights of the norm in front of what comes next, or null
    float eps2, offset2;
};

__device__ __forceinline__ int entry_row(const NormInput& in, size_t row, int k) {
    const int slot = in.entry_slot[row * in.top + k];
    return slot >= 0 && MG_GUARDED(residual_norm, MG_GUARD_ROW, slot, in.n_slots) ? slot : -1;
}

__device__ __forceinline__ float norm_input(const NormInput& in, size_t row, int width, int c) {
    if (in.entry_slot == nullptr) {
        const size_t i = row * width + c;
        return in.b ? fmaf(in.sb, in.b[i], in.sa * in.a[i]) : in.sa * in.a[i];
    }
    float sum = 0.f;
    for (int k = 0; k < in.top; ++k) {
        const int slot = entry_row(in, row, k);
        if (slot >= 0) sum += in.a[(size_t)slot * width + c];
    }
    return sum;
}

// The general form: one warp a row, two or three passes over the row (any width).
__global__ void __launch_bounds__(32 * NORM_WARPS)
norm_add_kernel(const NormInput in, const NormOutput out, int rows, int width) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x * NORM_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= rows) return;
    float mean = 0.f;
    if (out.center) {
        for (int c = lane; c < width; c += 32) mean += norm_input(in, row, width, c);
        mean = warp_sum(mean) / (float)width;
    }
    float sq = 0.f;
    for (int c = lane; c < width; c += 32) {
        const float y = norm_input(in, row, width, c) - mean;
        sq = fmaf(y, y, sq);
    }
    const float rstd = 1.0f / sqrtf(warp_sum(sq) / (float)width + out.eps);
    float sq2 = 0.f;
    for (int c = lane; c < width; c += 32) {
        const size_t i = (size_t)row * width + c;
        const float y = norm_input(in, row, width, c) - mean;
        const float x = out.x[i] + out.scale * (y * rstd * (out.offset + out.w[c]));
        out.x[i] = x;
        sq2 = fmaf(x, x, sq2);
        if (out.rows && !out.w2) out.rows[i] = __float2bfloat16_rn(x);
        if (out.clear) {
            in.a[i] = 0.f;
            if (in.b) in.b[i] = 0.f;
        }
    }
    if (!out.w2) return;
    const float r2 = 1.0f / sqrtf(warp_sum(sq2) / (float)width + out.eps2);
    for (int c = lane; c < width; c += 32) {               // (a lane reads what it wrote itself)
        const size_t i = (size_t)row * width + c;
        const float h = out.x[i] * r2 * (out.offset2 + out.w2[c]);
        if (out.rows) out.rows[i] = __float2bfloat16_rn(h);
        else out.rows32[i] = h;
    }
}

__device__ __forceinline__ float row_total(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_THREADS / 32; ++k) total += red[k];
    return total;
}

// The vector form: one CTA a row, the row's numbers asked for at once (16 bytes a load) and held in registers
// between the statistics and the sum, so that a step of few rows is one trip to memory and not a chain of them.
template <int ROW_VECS>       // float4 a thread holds: 1, 2, 4 or 8 (rows of up to 1,024 ... 8,192 numbers)
__global__ void __launch_bounds__(ROW_THREADS)
norm_add_vec_kernel(const NormInput in, const NormOutput out, int width) {
    __shared__ float red[2][ROW_THREADS / 32];
    pdl_trigger();
    pdl_wait();
    const int vecs = width >> 2, tid = threadIdx.x;
    const size_t row = blockIdx.x, base = row * vecs;
    float4* ar = reinterpret_cast<float4*>(in.a) + base;
    float4* br = in.b ? reinterpret_cast<float4*>(in.b) + base : nullptr;
    float4* xr = reinterpret_cast<float4*>(out.x) + base;
    const float4* wr = reinterpret_cast<const float4*>(out.w);
    float4 y[ROW_VECS], xv[ROW_VECS], wv[ROW_VECS];
#pragma unroll
    for (int u = 0; u < ROW_VECS; ++u) {
        const int i = tid + u * ROW_THREADS;
        y[u] = xv[u] = wv[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < vecs) {
            if (in.entry_slot == nullptr) {
                const float4 av = ar[i];
                y[u] = make_float4(in.sa * av.x, in.sa * av.y, in.sa * av.z, in.sa * av.w);
                if (br) {
                    const float4 bv = br[i];
                    y[u] = make_float4(fmaf(in.sb, bv.x, y[u].x), fmaf(in.sb, bv.y, y[u].y), fmaf(in.sb, bv.z, y[u].z), fmaf(in.sb, bv.w, y[u].w));
                }
            }
            xv[u] = xr[i];
            wv[u] = wr[i];
        }
    }
    if (in.entry_slot != nullptr) {
#pragma unroll 4
        for (int k = 0; k < in.top; ++k) {
            const int slot = entry_row(in, row, k);
            if (slot < 0) continue;
            const float4* tr = reinterpret_cast<const float4*>(in.a) + (size_t)slot * vecs;
#pragma unroll
            for (int u = 0; u < ROW_VECS; ++u) {
                const int i = tid + u * ROW_THREADS;
                if (i < vecs) {
                    const float4 av = tr[i];
                    y[u] = make_float4(y[u].x + av.x, y[u].y + av.y, y[u].z + av.z, y[u].w + av.w);
                }
            }
        }
    }
    if (out.center) {
        float sum = 0.f;
#pragma unroll
        for (int u = 0; u < ROW_VECS; ++u) sum += (y[u].x + y[u].y) + (y[u].z + y[u].w);
        const float mean = row_total(sum, red[0]) / (float)width;
#pragma unroll
        for (int u = 0; u < ROW_VECS; ++u)
            if (tid + u * ROW_THREADS < vecs) y[u] = make_float4(y[u].x - mean, y[u].y - mean, y[u].z - mean, y[u].w - mean);
    }
    float sq = 0.f;
#pragma unroll
    for (int u = 0; u < ROW_VECS; ++u) sq = fmaf(y[u].x, y[u].x, fmaf(y[u].y, y[u].y, fmaf(y[u].z, y[u].z, fmaf(y[u].w, y[u].w, sq))));
    const float rstd = 1.0f / sqrtf(row_total(sq, red[1]) / (float)width + out.eps);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float sc = out.scale, off = out.offset;
#pragma unroll
    for (int u = 0; u < ROW_VECS; ++u) {
        const int i = tid + u * ROW_THREADS;
        if (i < vecs) {
            const float4 r = make_float4(xv[u].x + sc * (y[u].x * rstd * (off + wv[u].x)), xv[u].y + sc * (y[u].y * rstd * (off + wv[u].y)),
                                         xv[u].z + sc * (y[u].z * rstd * (off + wv[u].z)), xv[u].w + sc * (y[u].w * rstd * (off + wv[u].w)));
            xr[i] = r;
            xv[u] = r;
            if (out.rows && !out.w2) {
                __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(out.rows + 4 * (base + i));
                o[0] = __floats2bfloat162_rn(r.x, r.y);
                o[1] = __floats2bfloat162_rn(r.z, r.w);
            }
            if (out.clear) {
                ar[i] = zero;
                if (br) br[i] = zero;
            }
        }
    }
    if (!out.w2) return;
    const float4* w2r = reinterpret_cast<const float4*>(out.w2);
    sq = 0.f;
#pragma unroll
    for (int u = 0; u < ROW_VECS; ++u) {
        sq = fmaf(xv[u].x, xv[u].x, fmaf(xv[u].y, xv[u].y, fmaf(xv[u].z, xv[u].z, fmaf(xv[u].w, xv[u].w, sq))));
        const int i = tid + u * ROW_THREADS;
        if (i < vecs) wv[u] = w2r[i];
    }
    const float r2 = 1.0f / sqrtf(row_total(sq, red[0]) / (float)width + out.eps2), off2 = out.offset2;
#pragma unroll
    for (int u = 0; u < ROW_VECS; ++u) {
        const int i = tid + u * ROW_THREADS;
        if (i < vecs) {
            const float a = xv[u].x * r2 * (off2 + wv[u].x), b = xv[u].y * r2 * (off2 + wv[u].y),
                        c = xv[u].z * r2 * (off2 + wv[u].z), d = xv[u].w * r2 * (off2 + wv[u].w);
            if (out.rows) store4(out.rows + 4 * (base + i), a, b, c, d);
            else store4(out.rows32 + 4 * (base + i), a, b, c, d);
        }
    }
}

__global__ void add_rows_kernel(float* __restrict__ x, const float* __restrict__ e, const float* __restrict__ v,
                                long long n, int width) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float y = x[i] + v[i % width];
    if (e) y += e[i];
    x[i] = y;
}

__global__ void scaled_sum_kernel(float* __restrict__ x, float* __restrict__ a, float sa, float* __restrict__ b, float sb,
                                  long long n, int clear) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    x[i] += fmaf(sb, b[i], sa * a[i]);
    if (clear) a[i] = b[i] = 0.f;
}

__global__ void softcap_kernel(float* x, long long n, float cap) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

template <typename T>
__global__ void cast_rows_kernel(const float* __restrict__ x, T* __restrict__ out, long long n, int use_tanh) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_float<T>(use_tanh ? tanhf(x[i]) : x[i]);
}

template <typename TW, typename T>
__global__ void token_gate_kernel(const float* __restrict__ g, const int* __restrict__ ids, const int* __restrict__ pos,
                                  const int* __restrict__ source, const int* __restrict__ previous,
                                  const TW* __restrict__ table, int table_ld, int off, T* __restrict__ out, int dim,
                                  int vocab, int n_previous) {
    pdl_trigger();
    pdl_wait();
    const int n = blockIdx.x;
    T* orow = out + (size_t)n * dim;
    if (pos[n] < 0) {
        for (int j = threadIdx.x; j < dim; j += blockDim.x) orow[j] = from_float<T>(0.f);
        return;
    }
    int id = ids[n];
    if (source != nullptr) {
        const int src = source[n];
        if (src >= 0 && MG_GUARDED(residual_norm, MG_GUARD_SOURCE, src, n_previous)) id = previous[src];
    }
    if (!MG_GUARDED(residual_norm, MG_GUARD_TOKEN, id, vocab)) id = 0;
    const TW* trow = table + (size_t)id * table_ld + off;
    const float* grow = g + (size_t)n * dim;
    for (int j = threadIdx.x; j < dim; j += blockDim.x) {
        const float z = grow[j];
        const float act = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
        orow[j] = from_float<T>(act * to_float(trow[j]));
    }
}

}  // namespace

// x: [rows, width] 32-bit, in place; a (and b, or null): [rows, width] 32-bit (zeroed if clear); w: [width] 32-bit.
// center: the row's mean is taken off first.  scale: factor on what is added.  out_rows: [rows, width] bfloat16 (32-bit
// if rows_32bit, only with w2) or null; w2 ([width] 32-bit or null), eps2, offset2: the norm that out_rows is of the new x.
// entry_slot (or null): [rows, top] rows of a, [n_slots, width], whose sum is the input (below zero: none); then b must be
// null and clear 0.
MG_API int mg_norm_add(float* x, float* a, float sa, float* b, float sb, const int* entry_slot, int top, int n_slots,
                       const float* w, int rows, int width, float eps, float offset, int center, float scale, int clear,
                       void* out_rows, int rows_32bit, const float* w2, float eps2, float offset2, void* stream) {
    if (rows == 0) return MG_OK;
    MG_REQUIRE(rows > 0 && width > 0 && x && a && w, "norm_add: bad sizes");
    MG_REQUIRE(entry_slot == nullptr || (top > 0 && n_slots > 0 && b == nullptr && !clear && sa == 1.f),
               "norm_add: a sum over entries takes neither a second input nor a factor, and is not cleared");
    MG_REQUIRE((w2 == nullptr || out_rows != nullptr) && (!rows_32bit || w2 != nullptr), "norm_add: rows that nothing is written to");
    const NormInput in{a, sa, b, sb, entry_slot, top, n_slots};
    const NormOutput out{x, w, eps, offset, scale, center, clear, rows_32bit ? nullptr : (bf16*)out_rows,
                         rows_32bit ? (float*)out_rows : nullptr, w2, eps2, offset2};
    const bool vec = width % 4 == 0 && width <= ROW_THREADS * MAX_ROW_VECS * 4 && (uintptr_t)x % 16 == 0 && (uintptr_t)a % 16 == 0 &&
                     (uintptr_t)b % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)out_rows % (w2 ? 16 : 4) == 0 && (uintptr_t)w2 % 16 == 0;
    const int per_thread = ceil_div(width / 4, ROW_THREADS);
    auto vec_kernel = per_thread <= 1 ? norm_add_vec_kernel<1> : per_thread <= 2 ? norm_add_vec_kernel<2>
                    : per_thread <= 4 ? norm_add_vec_kernel<4> : norm_add_vec_kernel<8>;
    const cudaError_t e =
        vec ? mg_launch(vec_kernel, dim3(rows), dim3(ROW_THREADS), 0, (cudaStream_t)stream, true, in, out, width)
            : mg_launch(norm_add_kernel, dim3(ceil_div(rows, NORM_WARPS)), dim3(32 * NORM_WARPS), 0, (cudaStream_t)stream,
                        true, in, out, rows, width);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "norm_add: %s", cudaGetErrorString(e));
    return MG_OK;
}

// x: [n / width, width] 32-bit, in place; e: the same shape or null; v: [width] 32-bit.
MG_API int mg_add_rows(float* x, const float* e, const float* v, long long n, int width, void* stream) {
    if (n == 0) return MG_OK;
    MG_REQUIRE(n > 0 && n < (1ll << 40) && width > 0 && n % width == 0 && v, "add_rows: bad sizes");
    const cudaError_t err = mg_launch(add_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0,
                                      (cudaStream_t)stream, true, x, e, v, n, width);
    if (err != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "add_rows: %s", cudaGetErrorString(err));
    return MG_OK;
}

MG_API int mg_scaled_sum(float* x, float* a, float sa, float* b, float sb, long long n, int clear, void* stream) {
    if (n == 0) return MG_OK;
    MG_REQUIRE(n > 0 && n < (1ll << 40) && a && b, "scaled_sum: bad sizes");
    const cudaError_t e = mg_launch(scaled_sum_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0,
                                    (cudaStream_t)stream, true, x, a, sa, b, sb, n, clear);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "scaled_sum: %s", cudaGetErrorString(e));
    return MG_OK;
}

MG_API int mg_softcap(float* x, long long n, float cap, void* stream) {
    if (n == 0) return MG_OK;
    MG_REQUIRE(n > 0 && n < (1ll << 40) && cap > 0.f, "softcap: bad size or cap");
    const cudaError_t e = mg_launch(softcap_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream,
                                    true, x, n, cap);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "softcap: %s", cudaGetErrorString(e));
    return MG_OK;
}

// out[i] = x[i], or tanh(x[i]) if use_tanh, in bfloat16 (out_bf16) or 32-bit (out may then be x itself).
MG_API int mg_cast_rows(const float* x, void* out, long long n, int use_tanh, int out_bf16, void* stream) {
    if (n == 0) return MG_OK;
    MG_REQUIRE(n > 0 && n < (1ll << 40), "cast: bad size");
    const dim3 grid((unsigned)((n + 255) / 256));
    const cudaError_t e =
        out_bf16 ? mg_launch(cast_rows_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, true, x, (bf16*)out, n, use_tanh)
                 : mg_launch(cast_rows_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, true, x, (float*)out, n, use_tanh);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "cast: %s", cudaGetErrorString(e));
    return MG_OK;
}

// g: [n_tokens, dim] 32-bit; table: [vocab, table_ld] (bfloat16 if table_bf16 else 32-bit), of which columns
// off .. off + dim - 1 are read; out: [n_tokens, dim] (bfloat16 if out_bf16 else 32-bit).  source / previous as in
// mg_embed; n_previous: ids that `previous` holds.
MG_API int mg_token_gate(const float* g, const int* ids, const int* pos, const int* source, const int* previous,
                         const void* table, int table_ld, int off, void* out, int n_tokens, int dim, int vocab,
                         int n_previous, int table_bf16, int out_bf16, void* stream) {
    if (n_tokens == 0) return MG_OK;
    MG_REQUIRE(n_tokens > 0 && dim > 0 && vocab > 0 && off >= 0 && off + dim <= table_ld, "token_gate: bad sizes");
    MG_REQUIRE(source == nullptr || previous != nullptr, "token_gate: token sources without the ids they point to");
    MG_REQUIRE(table_bf16 == out_bf16, "token_gate: the table and the output share a type");
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = dim >= 128 ? 128 : dim >= 64 ? 64 : 32;
    const cudaError_t e =
        out_bf16 ? mg_launch(token_gate_kernel<bf16, bf16>, dim3(n_tokens), dim3(threads), 0, s, true, g, ids, pos, source,
                             previous, (const bf16*)table, table_ld, off, (bf16*)out, dim, vocab, n_previous)
                 : mg_launch(token_gate_kernel<float, float>, dim3(n_tokens), dim3(threads), 0, s, true, g, ids, pos, source,
                             previous, (const float*)table, table_ld, off, (float*)out, dim, vocab, n_previous);
    if (e != cudaSuccess) return mg_set_error(MG_ERR_CUDA, "token_gate: %s", cudaGetErrorString(e));
    return MG_OK;
}
