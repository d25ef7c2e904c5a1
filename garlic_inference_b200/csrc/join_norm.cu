// A sublayer's result joins the residual stream through a norm of its own, and the stream goes on to the next reader,
// in one pass:
//
//   s = x + J(delta);  [x <- s];  out = L(s)
//
//   J (how the pending result joins): nothing pending; as it is; Dynamic Tanh tanh(alpha d) w + b; or RMS
//     d / sqrt(mean(d^2) + eps) * w
//   L (what the next reader gets): nothing; s rounded to the activation type (out may be columns of a wider matrix);
//     Dynamic Tanh of s; or RMS of s
//
// x is the float32 stream, delta and out have the activation type T, everything between is float32 and rounded once.
// With `rows` the input rows are picked and nothing is written back.  A row's result does not depend on what else is
// in the launch: thread count and slices follow from the width and the kinds alone, and sums run in a fixed order.
// Without an RMS no sum ties a row's elements together, so a row may be cut over several blocks; blocks walk several
// rows when there are many, so that the norms' vectors stay in the L1 cache.  Under bfloat16 tanh is 1 - 2 / (1 + e^2z)
// with the hardware's exponential and division (absolute error about 1e-7), under float32 the library's tanhf.
// NikolayBlagoev/garlic-inference adds its sublayers' results as they are (src/src-cuda/norm.cu:51-101).
#include "common.cuh"
#include <math.h>

#define JN_NONE 0
#define JN_PLAIN 1            // the result as it is / the stream as it is
#define JN_DYT 2
#define JN_RMS 3

struct JoinVecs {             // the vectors of one norm, in one type
    const void *w, *b, *alpha;
    int dtype;
    float eps;
};

template <typename T> __device__ __forceinline__ float jn_tanh(float z);
template <> __device__ __forceinline__ float jn_tanh<float>(float z) { return tanhf(z); }
template <> __device__ __forceinline__ float jn_tanh<bf16>(float z) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * fminf(z, 40.f))); }

template <typename T>
__device__ __forceinline__ float4 jn_dyt4(float4 z, float a, float4 w, float4 b) {
    return make_float4(fmaf(jn_tanh<T>(a * z.x), w.x, b.x), fmaf(jn_tanh<T>(a * z.y), w.y, b.y),
                       fmaf(jn_tanh<T>(a * z.z), w.z, b.z), fmaf(jn_tanh<T>(a * z.w), w.w, b.w));
}

// Four elements per thread and load; ITS such words of a row per thread.  Kinds without a sum: ITS = 1 and blockIdx.y
// is the row's slice.
template <typename T, int JOIN, int LAST, int ITS>
__global__ void __launch_bounds__(512)
join_norm_vec_kernel(const T* __restrict__ delta, JoinVecs j, float* __restrict__ residual, JoinVecs l, T* __restrict__ out,
                     long long ld_out, const int* __restrict__ rows, int n_rows, int dim, int write_residual) {
    gi_pdl_launch_dependents();
    __shared__ float red[33];
    const int c0 = (blockIdx.y * ITS * blockDim.x + threadIdx.x) * 4;
    const float ja = JOIN == JN_DYT ? load_w(j.alpha, j.dtype, 0) : 0.f;
    const float la = LAST == JN_DYT ? load_w(l.alpha, l.dtype, 0) : 0.f;
    // the first word's vectors are nobody's output: asked for before the wait
    float4 jw, jb, lw, lb;
    jw = jb = lw = lb = make_float4(0.f, 0.f, 0.f, 0.f);
    auto vectors = [&](int c) {
        if (JOIN >= JN_DYT) jw = load4_w(j.w, j.dtype, c);
        if (JOIN == JN_DYT) jb = load4_w(j.b, j.dtype, c);
        if (LAST >= JN_DYT) lw = load4_w(l.w, l.dtype, c);
        if (LAST == JN_DYT) lb = load4_w(l.b, l.dtype, c);
    };
    if (c0 < dim) vectors(c0);
    gi_pdl_wait();
    for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
        const size_t i = rows ? (size_t)rows[r] : (size_t)r;
        float* res = residual + i * dim;
        const T* del = delta + i * dim;
        float4 s[ITS], d[ITS];
        float sum = 0.f;
#pragma unroll
        for (int it = 0; it < ITS; ++it) {
            const int c = c0 + it * blockDim.x * 4;
            if (c < dim) {
                s[it] = load4_f32(res + c);
                if (JOIN != JN_NONE) d[it] = load4_act(del + c);
                if (JOIN == JN_RMS) { sum += d[it].x * d[it].x; sum += d[it].y * d[it].y; sum += d[it].z * d[it].z; sum += d[it].w * d[it].w; }
            }
        }
        const float j_inv = JOIN == JN_RMS ? 1.f / sqrtf(block_sum(sum, red) / (float)dim + j.eps) : 1.f;
        float sq = 0.f;
#pragma unroll
        for (int it = 0; it < ITS; ++it) {
            const int c = c0 + it * blockDim.x * 4;
            if (c < dim) {
                if (ITS > 1) vectors(c);
                float4 v = s[it];
                if (JOIN == JN_PLAIN) { v.x += d[it].x; v.y += d[it].y; v.z += d[it].z; v.w += d[it].w; }
                if (JOIN == JN_DYT) {
                    const float4 y = jn_dyt4<T>(d[it], ja, jw, jb);
                    v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w;
                }
                if (JOIN == JN_RMS) {
                    v.x = fmaf(d[it].x * j_inv, jw.x, v.x); v.y = fmaf(d[it].y * j_inv, jw.y, v.y);
                    v.z = fmaf(d[it].z * j_inv, jw.z, v.z); v.w = fmaf(d[it].w * j_inv, jw.w, v.w);
                }
                if (JOIN != JN_NONE && write_residual) *reinterpret_cast<float4*>(res + c) = v;
                if (LAST == JN_PLAIN) store4_act(out + r * ld_out + c, v);
                if (LAST == JN_DYT) store4_act(out + r * ld_out + c, jn_dyt4<T>(v, la, lw, lb));
                if (LAST == JN_RMS) { s[it] = v; sq += v.x * v.x; sq += v.y * v.y; sq += v.z * v.z; sq += v.w * v.w; }
            }
        }
        if (LAST == JN_RMS) {
            __syncthreads();
            const float inv = 1.f / sqrtf(block_sum(sq, red) / (float)dim + l.eps);
#pragma unroll
            for (int it = 0; it < ITS; ++it) {
                const int c = c0 + it * blockDim.x * 4;
                if (c < dim) {
                    if (ITS > 1) lw = load4_w(l.w, l.dtype, c);
                    store4_act(out + r * ld_out + c, make_float4(s[it].x * inv * lw.x, s[it].y * inv * lw.y, s[it].z * inv * lw.z, s[it].w * inv * lw.w));
                }
            }
        }
        if (JOIN == JN_RMS || LAST == JN_RMS) __syncthreads();            // `red` is used again by the next row
    }
}

// Any width, element by element; a block per row.
template <typename T>
__global__ void __launch_bounds__(256)
join_norm_kernel(const T* __restrict__ delta, int join, JoinVecs j, float* __restrict__ residual, int last, JoinVecs l,
                 T* __restrict__ out, long long ld_out, const int* __restrict__ rows, int dim, int write_residual) {
    gi_pdl_start();
    __shared__ float red[33];
    const int r = blockIdx.x;
    const size_t i = rows ? (size_t)rows[r] : (size_t)r;
    float* res = residual + i * dim;
    const T* del = delta + i * dim;
    float sum = 0.f;
    if (join == JN_RMS)
        for (int c = threadIdx.x; c < dim; c += blockDim.x) { const float v = to_f32(del[c]); sum += v * v; }
    float inv = 1.f;
    if (join == JN_RMS) inv = 1.f / sqrtf(block_sum(sum, red) / (float)dim + j.eps);
    const float ja = join == JN_DYT ? load_w(j.alpha, j.dtype, 0) : 0.f, la = last == JN_DYT ? load_w(l.alpha, l.dtype, 0) : 0.f;
    auto joined = [&](int c) {
        const float x = res[c];
        if (join == JN_NONE) return x;
        const float d = to_f32(del[c]);
        if (join == JN_DYT) return x + fmaf(jn_tanh<T>(ja * d), load_w(j.w, j.dtype, c), load_w(j.b, j.dtype, c));
        if (join == JN_RMS) return fmaf(d * inv, load_w(j.w, j.dtype, c), x);
        return x + d;
    };
    float l_inv = 1.f;
    if (last == JN_RMS) {
        float sq = 0.f;
        for (int c = threadIdx.x; c < dim; c += blockDim.x) { const float s = joined(c); sq += s * s; }
        __syncthreads();
        l_inv = 1.f / sqrtf(block_sum(sq, red) / (float)dim + l.eps);
    }
    T* o = out ? out + r * ld_out : nullptr;
    for (int c = threadIdx.x; c < dim; c += blockDim.x) {
        const float s = joined(c);
        if (join != JN_NONE && write_residual) res[c] = s;
        if (last == JN_PLAIN) o[c] = from_f32<T>(s);
        else if (last == JN_DYT) o[c] = from_f32<T>(fmaf(jn_tanh<T>(la * s), load_w(l.w, l.dtype, c), load_w(l.b, l.dtype, c)));
        else if (last == JN_RMS) o[c] = from_f32<T>(s * l_inv * load_w(l.w, l.dtype, c));
    }
}

template <typename T, int JOIN, int LAST>
static void launch_vec(const void* delta, const JoinVecs& j, float* residual, const JoinVecs& l, void* out, long long ld_out,
                       const int* rows, int n_rows, int dim, int write_residual, cudaStream_t s) {
    constexpr bool SUMS = JOIN == JN_RMS || LAST == JN_RMS;
    const int words = dim / 4;
    if (SUMS) {
        const int threads = words > 512 ? 512 : (words + 31) / 32 * 32;
        const int blocks = n_rows < 148 * 4 ? n_rows : 148 * 4;
        if (words <= threads)
            gi_launch(join_norm_vec_kernel<T, JOIN, LAST, 1>, dim3(blocks), dim3(threads), 0, s, (const T*)delta, j, residual, l,
                      (T*)out, ld_out, rows, n_rows, dim, write_residual);
        else if (words <= 2 * threads)
            gi_launch(join_norm_vec_kernel<T, JOIN, LAST, 2>, dim3(blocks), dim3(threads), 0, s, (const T*)delta, j, residual, l,
                      (T*)out, ld_out, rows, n_rows, dim, write_residual);
        else
            gi_launch(join_norm_vec_kernel<T, JOIN, LAST, 4>, dim3(blocks), dim3(threads), 0, s, (const T*)delta, j, residual, l,
                      (T*)out, ld_out, rows, n_rows, dim, write_residual);
    } else {
        const int threads = words > 256 ? 256 : (words + 31) / 32 * 32, slices = (words + threads - 1) / threads;
        const int most = 148 * 8 / slices > 0 ? 148 * 8 / slices : 1;
        gi_launch(join_norm_vec_kernel<T, JOIN, LAST, 1>, dim3(n_rows < most ? n_rows : most, slices), dim3(threads), 0, s,
                  (const T*)delta, j, residual, l, (T*)out, ld_out, rows, n_rows, dim, write_residual);
    }
}

template <typename T>
static int join_norm(const void* delta, int join, const JoinVecs& j, float* residual, int last, const JoinVecs& l, void* out,
                     long long ld_out, const int* rows, int n_rows, int dim, int write_residual, cudaStream_t s) {
    auto on16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    const bool vec = dim % 4 == 0 && dim <= 8192 && on16(delta) && on16(residual) && on16(j.w) && on16(j.b) && on16(l.w) && on16(l.b) &&
                     on16(out) && ld_out % 4 == 0;
    if (!vec) {
        gi_launch(join_norm_kernel<T>, dim3(n_rows), dim3(256), 0, s, (const T*)delta, join, j, residual, last, l, (T*)out, ld_out,
                  rows, dim, write_residual);
        return gi_check_launch("gi_join_norm");
    }
#define JN_CASE(J, L)                                                                                                   \
    if (join == J && last == L) {                                                                                       \
        launch_vec<T, J, L>(delta, j, residual, l, out, ld_out, rows, n_rows, dim, write_residual, s);                  \
        return gi_check_launch("gi_join_norm");                                                                         \
    }
#define JN_ROW(J) JN_CASE(J, JN_NONE) JN_CASE(J, JN_PLAIN) JN_CASE(J, JN_DYT) JN_CASE(J, JN_RMS)
    JN_ROW(JN_NONE) JN_ROW(JN_PLAIN) JN_ROW(JN_DYT) JN_ROW(JN_RMS)
#undef JN_ROW
#undef JN_CASE
    return 0;
}

extern "C" int gi_join_norm(const void* delta, int act_dtype, int join, const void* j_w, const void* j_b, const void* j_alpha,
                            int j_dtype, float j_eps, float* residual, int last, const void* l_w, const void* l_b,
                            const void* l_alpha, int l_dtype, float l_eps, void* out, long long ld_out, const int* rows,
                            int n_rows, int dim, int write_residual, void* stream) {
    GI_REQUIRE(n_rows >= 0 && dim > 0, "gi_join_norm: sizes must be positive");
    GI_REQUIRE(join >= JN_NONE && join <= JN_RMS && last >= JN_NONE && last <= JN_RMS, "gi_join_norm: kinds %d and %d", join, last);
    GI_REQUIRE((join == JN_NONE) == (delta == nullptr), "gi_join_norm: a pending result and how it joins come together");
    GI_REQUIRE(join < JN_DYT || (j_w && (join == JN_RMS || (j_b && j_alpha))), "gi_join_norm: the joining norm's vectors");
    GI_REQUIRE(last < JN_DYT || (l_w && (last == JN_RMS || (l_b && l_alpha))), "gi_join_norm: the last norm's vectors");
    GI_REQUIRE(last == JN_NONE || (out && ld_out >= dim), "gi_join_norm: output rows of %lld for %d elements", ld_out, dim);
    GI_REQUIRE(!(rows && write_residual), "gi_join_norm: gathered rows are never written back");
    if (n_rows == 0) return 0;
    const JoinVecs j = {j_w, j_b, j_alpha, j_dtype, j_eps}, l = {l_w, l_b, l_alpha, l_dtype, l_eps};
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == GI_DTYPE_F32)
        return join_norm<float>(delta, join, j, residual, last, l, out, ld_out, rows, n_rows, dim, write_residual, s);
    if (act_dtype == GI_DTYPE_BF16)
        return join_norm<bf16>(delta, join, j, residual, last, l, out, ld_out, rows, n_rows, dim, write_residual, s);
    GI_REQUIRE(false, "gi_join_norm: activation dtype %d", act_dtype);
}

// ------------------------------------------------------------------ a per-token input of a layer
// out[r, c] = gelu_tanh(z[r, c]) * table[tokens[r], off + c]: a gate made from the stream times the layer's own columns
// of a table that has a row per token of the vocabulary.  A token outside the table gives zeros.
template <typename T>
__global__ void token_side_gate_kernel(const T* __restrict__ z, const int* __restrict__ tokens, const void* __restrict__ table,
                                       int t_dtype, long long t_cols, int t_rows, int off, T* __restrict__ out, long long total,
                                       int dim) {
    gi_pdl_start();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / dim;
        const int c = (int)(i - r * dim), tok = tokens[r];
        float e = 0.f;
        if (tok >= 0 && tok < t_rows) {
            const long long at = tok * t_cols + off + c;
            e = t_dtype == GI_DTYPE_F32 ? ((const float*)table)[at] : to_f32(((const bf16*)table)[at]);
        }
        const float v = to_f32(z[i]);
        const float g = 0.5f * v * (1.f + jn_tanh<T>(0.7978845608028654f * (v + 0.044715f * v * v * v)));
        out[i] = from_f32<T>(g * e);
    }
}

extern "C" int gi_token_side_gate(const void* z, const int* tokens, const void* table, int t_dtype, int t_rows, int t_cols,
                                  int off, void* out, int act_dtype, int n_rows, int dim, void* stream) {
    GI_REQUIRE(n_rows >= 0 && dim > 0 && t_rows > 0 && off >= 0 && off + dim <= t_cols, "gi_token_side_gate: columns %d .. %d of %d",
               off, off + dim, t_cols);
    GI_REQUIRE(t_dtype == GI_DTYPE_F32 || t_dtype == GI_DTYPE_BF16, "gi_token_side_gate: table dtype %d", t_dtype);
    if (n_rows == 0) return 0;
    const long long total = (long long)n_rows * dim;
    const int blocks = (int)((total + 255) / 256 > 148 * 8 ? 148 * 8 : (total + 255) / 256);
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == GI_DTYPE_F32)
        gi_launch(token_side_gate_kernel<float>, dim3(blocks), dim3(256), 0, s, (const float*)z, tokens, table, t_dtype, (long long)t_cols,
                  t_rows, off, (float*)out, total, dim);
    else if (act_dtype == GI_DTYPE_BF16)
        gi_launch(token_side_gate_kernel<bf16>, dim3(blocks), dim3(256), 0, s, (const bf16*)z, tokens, table, t_dtype, (long long)t_cols,
                  t_rows, off, (bf16*)out, total, dim);
    else
        GI_REQUIRE(false, "gi_token_side_gate: activation dtype %d", act_dtype);
    return gi_check_launch("gi_token_side_gate");
}
