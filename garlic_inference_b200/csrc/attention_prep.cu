// The two ends of an attention mixer whose keys and values have shapes of their own, around the attention
// kernel itself.
//
//   gi_attn_prepare   per token: rotate the first n_rot dimensions of every query and key head by position x
//                     frequency (pairs (2r, 2r+1), or (r, r + n_rot/2) in the half layout; the angle is the float32
//                     product and its cosine and sine are taken here, so no table limits the positions), write the
//                     queries as [n, query rows, d] and put the token's keys and values into its cache page.  The
//                     inputs are columns of one wider matrix (a packed projection, or the output of the short
//                     convolutions, which is float32 whatever the activation type is).  With n_rot = 0 nothing
//                     turns; with k_off < 0 the layer has no keys and values of its own (it reads another layer's)
//                     and only the queries are written.  Before the rotation, optionally: a bias per column (`bias`,
//                     laid out [queries | keys | values] like the columns themselves); an RMS norm of all query
//                     columns of the token at once and another of all its key columns, each with a weight per column
//                     (`norm_w`, [queries | keys]; x / sqrt(mean(x^2) + eps) * w); and a factor on the queries that
//                     grows with the position p, 1 + temp_coef ln(floor((p + 1) / temp_every) + 1).  All float32.
//                     Cosine and sine may both be multiplied by a `magnitude`.  After the rotation, optionally
//                     (`head_eps` > 0): every query and key head is divided by its own root mean square over its d
//                     dimensions (eps inside the root, no weight).  With that option and the half layout (or no rotation)
//                     and widths that fit, a second kernel runs: a group of lanes per head, four elements per access.
//                     Optionally (`pool_block` P > 0): a token that completes a block of P positions also leaves the
//                     mean of the block's P keys, and of its P values, as the cache holds them (float32 sum, one
//                     rounding), as one row of the pools of block means.  For steps that bring one token of a
//                     sequence, where the block's other rows lie in the cache already; steps with several tokens run
//   gi_pool_blocks    afterwards, which does the same for every block that a token of the step completes.
//   gi_attn_finish    per token and head: o = a_1 - lam a_2 for mixers with two softmax maps per head (lam one
//                     number on the device), o = a_1 otherwise; optionally o / sqrt(mean(o^2) + eps); times a
//                     constant; times sigmoid(gate logit of the head, or of the head's element); rounded once into the
//                     activation type.
//
// Key pools are [pages, key heads, page_size, d], value pools [pages, value heads, page_size, dv].
// NikolayBlagoev/garlic-inference rotates by table and appends equal-shaped keys and values
// (src/src-cuda/rope.cu:41-79, src/src-cuda/kvcache.cu:61-84).
#include "common.cuh"
#include <math.h>

// The means of whole blocks of `block` positions: row b of a sequence lies in page b / rows of its row of `table`, at
// row b % rows of that page; pools [pages, heads, rows, d].  block = 0: none are kept.
struct BlockMeans {
    void *k, *v;
    const int* table;
    int block, rows, max_pages, n_pages;
};

// The block that ends at `pos` (pos + 1 is a multiple of its length), summed in the order of its positions, so that
// the row is the same whoever makes it.  Called by a whole thread block.
template <typename T>
__device__ __forceinline__ void pool_block(const T* k_pool, const T* v_pool, const int* __restrict__ bt_row, int pos,
                                           int slot, const BlockMeans& m, int n_kh, int n_vh, int d, int dv, int page_size,
                                           int max_pages, int n_pool_pages, int* __restrict__ status) {
    const int b = pos / m.block, lp = b / m.rows;
    const int to = lp < m.max_pages ? m.table[(size_t)slot * m.max_pages + lp] : -1;
    if (to < 0 || to >= m.n_pages) {
        if (threadIdx.x == 0) atomicExch(status, lp < m.max_pages ? 2 : 1);
        return;
    }
    const float share = 1.f / (float)m.block;
    const int first = b * m.block, row = b - lp * m.rows;
    const int lp0 = first / page_size, in0 = first - lp0 * page_size;      // page and row of the block's first position
    constexpr int N = 16 / (int)sizeof(T);                                 // elements of a 16-byte word
    const bool wide = d % N == 0 && dv % N == 0;
    const int step = wide ? N : 1;
    const int nk = n_kh * d / step, nv = n_vh * dv / step;
    for (int i = threadIdx.x; i < nk + nv; i += blockDim.x) {
        const bool key = i < nk;
        const int w = key ? d : dv, heads = key ? n_kh : n_vh, e = (key ? i : i - nk) * step;
        const int h = e / w, c = e - h * w;
        const T* pool = key ? k_pool : v_pool;
        T* out = (T*)(key ? m.k : m.v) + (((size_t)to * heads + h) * m.rows + row) * w + c;
        float sum[N];
#pragma unroll
        for (int x = 0; x < N; ++x) sum[x] = 0.f;
        int tp = lp0, in = in0;
        for (int p0 = 0; p0 < m.block; p0 += 8) {                          // eight positions under way at a time
            size_t at[8];
            bool ok[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const bool want = p0 + u < m.block;
                const int page = want && tp < max_pages ? bt_row[tp] : -1;
                ok[u] = page >= 0 && page < n_pool_pages;
                if (want && !ok[u]) atomicExch(status, 5);
                at[u] = (((size_t)(ok[u] ? page : 0) * heads + h) * page_size + in) * w + c;
                if (++in == page_size) { in = 0; ++tp; }
            }
            if (wide) {
                uint4 v[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) if (ok[u]) v[u] = *reinterpret_cast<const uint4*>(pool + at[u]);
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const T* x4 = reinterpret_cast<const T*>(&v[u]);
                    if (ok[u]) {
#pragma unroll
                        for (int x = 0; x < N; ++x) sum[x] += to_f32(x4[x]);
                    }
                }
            } else {
#pragma unroll
                for (int u = 0; u < 8; ++u) if (ok[u]) sum[0] += to_f32(pool[at[u]]);
            }
        }
        if (wide) {
            uint4 o;
            T* o4 = reinterpret_cast<T*>(&o);
#pragma unroll
            for (int x = 0; x < N; ++x) o4[x] = from_f32<T>(sum[x] * share);
            *reinterpret_cast<uint4*>(out) = o;
        } else {
            *out = from_f32<T>(sum[0] * share);
        }
    }
}

template <typename TI, typename T, bool MEANS>
__global__ void attn_prepare_kernel(const TI* __restrict__ src, long long ld, int q_off, int k_off, int v_off,
                                    const float* __restrict__ freq, int n_rot, int half_layout,
                                    const int* __restrict__ tok_pos, const int* __restrict__ tok_slot,
                                    const int* __restrict__ block_table, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                    T* __restrict__ q_out, int n_qh, int n_kh, int n_vh, int d, int dv, int page_size,
                                    int max_pages, int n_pool_pages, int append, int* __restrict__ status,
                                    const void* __restrict__ bias, int bias_dtype, const void* __restrict__ norm_w,
                                    int norm_dtype, float norm_eps, float temp_coef, int temp_every, BlockMeans means,
                                    float magnitude, float head_eps) {
    gi_pdl_start();
    extern __shared__ float cs[];                 // cos [n_rot/2], sin [n_rot/2], a factor per query and key head
    __shared__ float red[33];
    const int t = blockIdx.x;
    const int slot = tok_slot[t], pos = tok_pos[t];
    const TI* row = src + (size_t)t * ld;
    const int pairs = n_rot / 2;
    const int nq = n_qh * d, nk = k_off >= 0 ? n_kh * d : 0;
    // element i of the token's queries (i < nq) or keys (i - nq) as float32, with its bias
    auto raw = [&](int i) {
        const float x = to_f32(row[i < nq ? q_off + i : k_off + (i - nq)]);
        return bias ? x + load_w(bias, bias_dtype, i) : x;
    };
    float q_mul = 1.f, k_mul = 1.f;
    if (norm_w) {
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < nq; i += blockDim.x) { const float x = raw(i); sq = fmaf(x, x, sq); }
        for (int i = nq + threadIdx.x; i < nq + nk; i += blockDim.x) { const float x = raw(i); sk = fmaf(x, x, sk); }
        sq = block_sum(sq, red);
        __syncthreads();
        sk = block_sum(sk, red);
        q_mul = 1.f / sqrtf(sq / (float)nq + norm_eps);
        if (nk) k_mul = 1.f / sqrtf(sk / (float)nk + norm_eps);
    }
    if (temp_every > 0) q_mul *= 1.f + temp_coef * logf((float)((max(pos, 0) + 1) / temp_every) + 1.f);
    // the same element as the attention reads it: normed, weighted, and (queries) times the position's factor
    auto val = [&](int i) {
        const float x = raw(i) * (i < nq ? q_mul : k_mul);
        return norm_w ? x * load_w(norm_w, norm_dtype, i) : x;
    };
    for (int r = threadIdx.x; r < pairs; r += blockDim.x) {
        float s, c;
        sincosf((float)pos * freq[r], &s, &c);
        cs[r] = c * magnitude;
        cs[pairs + r] = s * magnitude;
    }
    __syncthreads();
    const int heads = n_qh + (k_off >= 0 ? n_kh : 0), rest = d - n_rot;
    float* hm = cs + n_rot;                       // 1 / root mean square of every head after its rotation
    if (head_eps > 0.f) {
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
        for (int h = warp; h < heads; h += blockDim.x >> 5) {
            float sum = 0.f;
            for (int r = lane; r < pairs; r += 32) {
                const int a = half_layout ? r : 2 * r, b = half_layout ? r + pairs : 2 * r + 1;
                const float u = val(h * d + a), v = val(h * d + b), c = cs[r], s = cs[pairs + r];
                const float ua = u * c - v * s, vb = v * c + u * s;
                sum += ua * ua + vb * vb;
            }
            for (int i = lane; i < rest; i += 32) { const float x = val(h * d + n_rot + i); sum += x * x; }
            sum = warp_sum(sum);
            if (lane == 0) hm[h] = 1.f / sqrtf(sum / (float)d + head_eps);
        }
        __syncthreads();
    }
    // where this token's keys and values go
    long long page = -1;
    if (append && k_off >= 0 && slot >= 0) {
        if (pos < 0 || pos / page_size >= max_pages) {
            if (threadIdx.x == 0) atomicExch(status, 1);
        } else {
            page = block_table[(size_t)slot * max_pages + pos / page_size];
            if (page < 0 || page >= n_pool_pages) {
                if (threadIdx.x == 0) atomicExch(status, 2);
                page = -1;
            }
        }
    }
    const int in_page = pos >= 0 ? pos % page_size : 0;
    // rotated pairs of the query and key heads
    for (int i = threadIdx.x; i < heads * pairs; i += blockDim.x) {
        const int h = i / pairs, r = i - h * pairs;
        const int a = half_layout ? r : 2 * r, b = half_layout ? r + pairs : 2 * r + 1;
        const bool is_q = h < n_qh;
        const float u = val(h * d + a), v = val(h * d + b);
        const float c = cs[r], s = cs[pairs + r];
        float ua = u * c - v * s, vb = v * c + u * s;
        if (head_eps > 0.f) { ua *= hm[h]; vb *= hm[h]; }
        if (is_q) {
            T* o = q_out + ((size_t)t * n_qh + h) * d;
            o[a] = from_f32<T>(ua);
            o[b] = from_f32<T>(vb);
        } else if (page >= 0) {
            T* o = k_pool + ((page * n_kh + (h - n_qh)) * page_size + in_page) * d;
            o[a] = from_f32<T>(ua);
            o[b] = from_f32<T>(vb);
        }
    }
    // the dimensions that pass
    for (int i = threadIdx.x; i < heads * rest; i += blockDim.x) {
        const int h = i / rest, c = n_rot + (i - h * rest);
        const bool is_q = h < n_qh;
        float x = val(h * d + c);
        if (head_eps > 0.f) x *= hm[h];
        if (is_q) q_out[((size_t)t * n_qh + h) * d + c] = from_f32<T>(x);
        else if (page >= 0) k_pool[((page * n_kh + (h - n_qh)) * page_size + in_page) * d + c] = from_f32<T>(x);
    }
    if (page >= 0) {
        for (int i = threadIdx.x; i < n_vh * dv; i += blockDim.x) {
            const int h = i / dv, c = i - h * dv;
            const float x = to_f32(row[v_off + i]);
            v_pool[((page * n_vh + h) * page_size + in_page) * dv + c] =
                from_f32<T>(bias ? x + load_w(bias, bias_dtype, nq + nk + i) : x);
        }
        if (MEANS && (pos + 1) % means.block == 0) {
            __syncthreads();                      // this token's own key and value are in the cache for the whole block
            pool_block<T>(k_pool, v_pool, block_table + (size_t)slot * max_pages, pos, slot, means, n_kh, n_vh, d, dv,
                          page_size, max_pages, n_pool_pages, status);
        }
    }
}

// The same for heads that are divided by their root mean square: a group of LPH lanes per head, every access four
// neighbouring elements.  A query's or key's words are its rotated pairs of words (4 dimensions and their 4 partners, half
// layout) and then the words that pass; lane i of the group owns pair or word i.  A value's words are the lanes' in pairs
// too (v_second: how far the second lies behind the first, 0 for widths that are no multiple of 8).  A block takes TOK tokens (their angles made once, before
// the wait) and walks the heads (queries, keys, values) that its place on the grid's second axis gives it; a head's bias
// is read once for all its tokens.  A head's result depends on its own row alone.
#define APH_THREADS 256
// 1 / sqrt: the hardware's approximation where the result is rounded to bfloat16
template <typename T> __device__ __forceinline__ float aph_inv_root(float x) { return 1.f / sqrtf(x); }
template <> __device__ __forceinline__ float aph_inv_root<bf16>(float x) { return rsqrtf(x); }

template <typename TI, typename T, int TOK, int LPH>
__global__ void __launch_bounds__(APH_THREADS)
attn_prepare_heads_kernel(const TI* __restrict__ src, long long ld, int q_off, int k_off, int v_off,
                          const float* __restrict__ freq, int n_rot, const int* __restrict__ tok_pos,
                          const int* __restrict__ tok_slot, const int* __restrict__ block_table, T* __restrict__ k_pool,
                          T* __restrict__ v_pool, T* __restrict__ q_out, int n_tokens, int n_qh, int n_kh, int n_vh, int d,
                          int dv, int page_size, int max_pages, int n_pool_pages, int append, int* __restrict__ status,
                          const void* __restrict__ bias, int bias_dtype, float magnitude, float head_eps, int lph_, int v_second) {
    gi_pdl_launch_dependents();
    extern __shared__ __align__(16) float cs[];   // per token cos [n_rot/2], sin [n_rot/2]
    __shared__ int page_of[TOK], row_of[TOK];     // where each token's key and value go; page -1: nowhere
    const int t0 = blockIdx.x * TOK, pairs = n_rot / 2;
    for (int i = threadIdx.x; i < TOK * pairs; i += APH_THREADS) {
        const int k = i / pairs, r = i - k * pairs;
        float s = 0.f, c = 1.f;
        if (t0 + k < n_tokens) sincosf((float)tok_pos[t0 + k] * freq[r], &s, &c);
        cs[k * n_rot + r] = c * magnitude;
        cs[k * n_rot + pairs + r] = s * magnitude;
    }
    if (threadIdx.x < TOK) {
        int to = -1, in = 0;
        const int t = t0 + threadIdx.x;
        if (t < n_tokens && append && k_off >= 0 && tok_slot[t] >= 0) {
            const int pos = tok_pos[t], lp = pos >= 0 ? pos / page_size : max_pages;
            if (lp >= max_pages) {
                if (blockIdx.y == 0) atomicExch(status, 1);
            } else {
                const int page = block_table[(size_t)tok_slot[t] * max_pages + lp];
                if (page < 0 || page >= n_pool_pages) {
                    if (blockIdx.y == 0) atomicExch(status, 2);
                } else {
                    to = page;
                    in = pos - lp * page_size;
                }
            }
        }
        page_of[threadIdx.x] = to;
        row_of[threadIdx.x] = in;
    }
    __syncthreads();
    gi_pdl_wait();
    const int lph = LPH > 0 ? LPH : lph_;
    const int groups = APH_THREADS / lph, group = threadIdx.x / lph, lane = threadIdx.x - group * lph;
    const int pair_words = pairs / 4, words = pair_words + (d - n_rot) / 4;
    const int qk = n_qh + (k_off >= 0 ? n_kh : 0), heads = qk + (k_off >= 0 ? n_vh : 0);
    const float share = 1.f / (float)d;
    const int n_here = min(TOK, n_tokens - t0);
    for (int h0 = blockIdx.y * groups; h0 < heads; h0 += gridDim.y * groups) {
        const int h = h0 + group;                 // a group past the last head walks along for the shuffles
        const bool is_v = h >= qk;
        // the lane's word inside its head, and how far its second word lies behind it (0: there is none)
        const int at = is_v || lane < pair_words ? 4 * lane : n_rot + 4 * (lane - pair_words);
        const int second = is_v ? v_second : (lane < pair_words ? pairs : 0);
        const bool mine = h < heads && lane < (is_v ? (v_second ? dv / 8 : dv / 4) : words), two = mine && second > 0;
        const bool turns = two && !is_v;
        const int col = is_v ? v_off + (h - qk) * dv : (h < n_qh ? q_off + h * d : k_off + (h - n_qh) * d);
        float4 ba = make_float4(0.f, 0.f, 0.f, 0.f), bb = ba;
        if (bias && mine) {
            const int b0 = (is_v ? qk * d + (h - qk) * dv : h * d) + at;
            ba = load4_w(bias, bias_dtype, b0);
            if (two) bb = load4_w(bias, bias_dtype, b0 + second);
        }
        const TI* p = src + (size_t)t0 * ld + col + at;
        float4 ua[TOK], ub[TOK];
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
            ua[k] = ub[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (k < n_here) {
                if (mine) ua[k] = load4_act(p + k * ld);
                if (two) ub[k] = load4_act(p + k * ld + second);
            }
        }
        // the head's rows: queries lie n_qh d apart, a key or value in the token's page
        T* const base = is_v ? v_pool : (h < n_qh ? q_out + ((size_t)t0 * n_qh + h) * d : k_pool);
        const int pool_heads = is_v ? n_vh : n_kh, pool_head = is_v ? h - qk : h - n_qh, wide = is_v ? dv : d;
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
            float4 a = make_float4(ua[k].x + ba.x, ua[k].y + ba.y, ua[k].z + ba.z, ua[k].w + ba.w);
            float4 b = make_float4(ub[k].x + bb.x, ub[k].y + bb.y, ub[k].z + bb.z, ub[k].w + bb.w);
            if (turns) {
                const float4 c = *reinterpret_cast<const float4*>(cs + k * n_rot + at);
                const float4 s = *reinterpret_cast<const float4*>(cs + k * n_rot + pairs + at);
                const float4 u = a, v = b;
                a = make_float4(u.x * c.x - v.x * s.x, u.y * c.y - v.y * s.y, u.z * c.z - v.z * s.z, u.w * c.w - v.w * s.w);
                b = make_float4(v.x * c.x + u.x * s.x, v.y * c.y + u.y * s.y, v.z * c.z + u.z * s.z, v.w * c.w + u.w * s.w);
            }
            float sum = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;      // words that are not the lane's are zeros
            sum += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
#pragma unroll
            for (int o = LPH > 0 ? LPH / 2 : 16; o > 0; o >>= 1)
                if (LPH > 0 || o < lph) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            const float m = is_v ? 1.f : aph_inv_root<T>(sum * share + head_eps);
            a.x *= m; a.y *= m; a.z *= m; a.w *= m;
            b.x *= m; b.y *= m; b.z *= m; b.w *= m;
            if (mine && k < n_here) {
                T* dst = base + (size_t)k * n_qh * d + at;
                bool there = true;
                if (h >= n_qh) {
                    const int page = page_of[k];
                    there = page >= 0;
                    dst = base + (((size_t)page * pool_heads + pool_head) * page_size + row_of[k]) * wide + at;
                }
                if (there) {
                    store4_act(dst, a);
                    if (two) store4_act(dst + second, b);
                }
            }
        }
    }
}

template <typename T>
__global__ void pool_blocks_kernel(const T* __restrict__ k_pool, const T* __restrict__ v_pool,
                                   const int* __restrict__ block_table, const int* __restrict__ tok_pos,
                                   const int* __restrict__ tok_slot, int n_kh, int n_vh, int d, int dv, int page_size,
                                   int max_pages, int n_pool_pages, int* __restrict__ status, BlockMeans means) {
    gi_pdl_start();
    const int slot = tok_slot[blockIdx.x], pos = tok_pos[blockIdx.x];
    if (slot < 0 || pos < 0 || (pos + 1) % means.block) return;
    pool_block<T>(k_pool, v_pool, block_table + (size_t)slot * max_pages, pos, slot, means, n_kh, n_vh, d, dv, page_size,
                  max_pages, n_pool_pages, status);
}

extern "C" int gi_pool_blocks(const void* k_pool, const void* v_pool, int act_dtype, const int* block_table,
                              const int* tok_pos, const int* tok_slot, int n_tokens, int n_kh, int n_vh, int d, int dv,
                              int page_size, int max_pages, int n_pool_pages, int* status, void* mean_k, void* mean_v,
                              const int* mean_table, int block, int mean_rows, int mean_max_pages, int mean_pages,
                              void* stream) {
    GI_REQUIRE(n_tokens >= 0 && n_kh > 0 && n_vh > 0 && d > 0 && dv > 0 && page_size > 0 && max_pages > 0, "gi_pool_blocks: sizes must be positive");
    GI_REQUIRE(block > 0 && mean_rows > 0 && mean_max_pages > 0 && mean_pages > 0, "gi_pool_blocks: blocks of %d positions", block);
    if (n_tokens == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const BlockMeans m = {mean_k, mean_v, mean_table, block, mean_rows, mean_max_pages, mean_pages};
    const int work = n_kh * d + n_vh * dv, threads = work >= 1024 ? 256 : 128;
    if (act_dtype == GI_DTYPE_F32)
        gi_launch(pool_blocks_kernel<float>, dim3(n_tokens), dim3(threads), 0, s, (const float*)k_pool, (const float*)v_pool,
                  block_table, tok_pos, tok_slot, n_kh, n_vh, d, dv, page_size, max_pages, n_pool_pages, status, m);
    else if (act_dtype == GI_DTYPE_BF16)
        gi_launch(pool_blocks_kernel<bf16>, dim3(n_tokens), dim3(threads), 0, s, (const bf16*)k_pool, (const bf16*)v_pool,
                  block_table, tok_pos, tok_slot, n_kh, n_vh, d, dv, page_size, max_pages, n_pool_pages, status, m);
    else
        GI_REQUIRE(false, "gi_pool_blocks: activation dtype %d", act_dtype);
    return gi_check_launch("gi_pool_blocks");
}

extern "C" int gi_attn_prepare(const void* src, int src_dtype, long long ld, int q_off, int k_off, int v_off,
                               const float* freq, int n_rot, int half_layout, const int* tok_pos, const int* tok_slot,
                               const int* block_table, void* k_pool, void* v_pool, void* q_out, int act_dtype,
                               int n_tokens, int n_qh, int n_kh, int n_vh, int d, int dv, int page_size, int max_pages,
                               int n_pool_pages, int append, int* status, const void* bias, int bias_dtype,
                               const void* norm_w, int norm_dtype, float norm_eps, float temp_coef, int temp_every,
                               void* mean_k, void* mean_v, const int* mean_table, int mean_block, int mean_rows,
                               int mean_max_pages, int mean_pages, float magnitude, float head_eps, void* stream) {
    GI_REQUIRE(head_eps >= 0.f && magnitude > 0.f, "gi_attn_prepare: the heads' eps and the factor on cosine and sine");
    GI_REQUIRE(n_tokens >= 0 && n_qh > 0 && d > 0 && dv > 0, "gi_attn_prepare: sizes must be positive");
    GI_REQUIRE(temp_every >= 0 && (!norm_w || norm_eps > 0.f), "gi_attn_prepare: the queries' factor and the norm's eps");
    GI_REQUIRE(n_rot >= 0 && n_rot % 2 == 0 && n_rot <= d, "gi_attn_prepare: %d rotated dimensions of heads of %d", n_rot, d);
    GI_REQUIRE(k_off < 0 || (n_kh > 0 && n_vh > 0 && page_size > 0 && max_pages > 0), "gi_attn_prepare: key/value sizes");
    GI_REQUIRE(mean_block == 0 || (mean_block > 0 && k_off >= 0 && append && mean_rows > 0 && mean_max_pages > 0 && mean_pages > 0),
               "gi_attn_prepare: means of blocks of %d positions", mean_block);
    const BlockMeans means = {mean_k, mean_v, mean_table, mean_block, mean_rows, mean_max_pages, mean_pages};
    if (n_tokens == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    // heads divided by their root mean square: a group of lanes per head, when every word of four elements falls into place
    if (head_eps > 0.f && (half_layout || n_rot == 0) && !norm_w && temp_every == 0 && mean_block == 0 && n_rot % 8 == 0 &&
        d % 4 == 0 && dv % 4 == 0) {
        const int esz = src_dtype == GI_DTYPE_F32 ? 4 : 2, ez = act_dtype == GI_DTYPE_F32 ? 4 : 2;
        const int words = n_rot / 8 + (d - n_rot) / 4, v_second = dv % 8 == 0 ? dv / 2 : 0;
        const int v_words = v_second ? dv / 8 : dv / 4, most = k_off >= 0 && v_words > words ? v_words : words;
        int lph = 1;
        while (lph < most) lph *= 2;
        const bool on_words = ld % 4 == 0 && q_off % 4 == 0 && (k_off < 0 || (k_off % 4 == 0 && v_off % 4 == 0)) &&
                              (uintptr_t)src % (4 * esz) == 0 && (uintptr_t)q_out % (4 * ez) == 0 && (uintptr_t)k_pool % (4 * ez) == 0 &&
                              (uintptr_t)v_pool % (4 * ez) == 0 && (uintptr_t)bias % 16 == 0;
        if (lph <= 32 && on_words) {
            const int heads = n_qh + (k_off >= 0 ? n_kh + n_vh : 0), groups = APH_THREADS / lph;
            const int rounds = (heads + groups - 1) / groups;
#define APH_LAUNCH(TI, T, TOK)                                                                                       \
            gi_launch(lph == 16 ? attn_prepare_heads_kernel<TI, T, TOK, 16> : attn_prepare_heads_kernel<TI, T, TOK, 0>, dim3((n_tokens + TOK - 1) / TOK, TOK > 1 ? (rounds + 1) / 2 : rounds),  \
                      dim3(APH_THREADS), (size_t)TOK * n_rot * sizeof(float), s, (const TI*)src, ld, q_off, k_off, v_off, freq,  \
                      n_rot, tok_pos, tok_slot, block_table, (T*)k_pool, (T*)v_pool, (T*)q_out, n_tokens, n_qh, n_kh, n_vh, d,  \
                      dv, page_size, max_pages, n_pool_pages, append, status, bias, bias_dtype, magnitude, head_eps, lph, v_second)
#define APH_TOK(TI, T) if (n_tokens >= 256) APH_LAUNCH(TI, T, 4); else APH_LAUNCH(TI, T, 1)
            if (src_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_F32) { APH_TOK(float, float); }
            else if (src_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_BF16) { APH_TOK(float, bf16); }
            else if (src_dtype == GI_DTYPE_BF16 && act_dtype == GI_DTYPE_BF16) { APH_TOK(bf16, bf16); }
            else GI_REQUIRE(false, "gi_attn_prepare: source dtype %d with activation dtype %d", src_dtype, act_dtype);
#undef APH_TOK
#undef APH_LAUNCH
            return gi_check_launch("gi_attn_prepare");
        }
    }
    const int n_heads = n_qh + (k_off >= 0 ? n_kh : 0);
    const size_t smem = (size_t)(n_rot + (head_eps > 0.f ? n_heads : 0)) * sizeof(float);
    GI_REQUIRE(smem <= 40 * 1024, "gi_attn_prepare: %d heads of which %d dimensions turn", n_heads, n_rot);
    const int work = (n_qh + (k_off >= 0 ? n_kh : 0)) * d;
    const int threads = work >= 2048 ? 256 : 128;
#define AP_LAUNCH(TI, T)                                                                                             \
    gi_launch(mean_block > 0 ? attn_prepare_kernel<TI, T, true> : attn_prepare_kernel<TI, T, false>, dim3(n_tokens), dim3(threads), smem, s, (const TI*)src, ld, q_off, k_off,   \
              v_off, freq, n_rot, half_layout, tok_pos, tok_slot, block_table, (T*)k_pool, (T*)v_pool, (T*)q_out,     \
              n_qh, n_kh, n_vh, d, dv, page_size, max_pages, n_pool_pages, append, status, bias, bias_dtype, norm_w,     \
              norm_dtype, norm_eps, temp_coef, temp_every, means, magnitude, head_eps)
    if (src_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_F32) AP_LAUNCH(float, float);
    else if (src_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_BF16) AP_LAUNCH(float, bf16);
    else if (src_dtype == GI_DTYPE_BF16 && act_dtype == GI_DTYPE_BF16) AP_LAUNCH(bf16, bf16);
    else GI_REQUIRE(false, "gi_attn_prepare: source dtype %d with activation dtype %d", src_dtype, act_dtype);
#undef AP_LAUNCH
    return gi_check_launch("gi_attn_prepare");
}

// att float32 [n, heads * maps, dv] (a head's maps side by side); gate: logit of head h at gate[r * ldg + h], or with
// gate_elems of its element c at gate[r * ldg + h * dv + c];
// out [n, ld_out] gets the head's dv values at column h * dv.
template <typename TA, typename T>
__global__ void attn_finish_kernel(const TA* __restrict__ att, int maps, const float* __restrict__ lam, float eps,
                                   int norm, float mul, const T* __restrict__ gate, long long ldg,
                                   T* __restrict__ out, long long ld_out, int heads, int dv, int gate_elems) {
    gi_pdl_start();
    __shared__ float red[33];
    const size_t r = blockIdx.x;
    const int h = blockIdx.y;
    const TA* a1 = att + (r * heads + h) * (size_t)maps * dv;
    const float l = maps > 1 ? lam[0] : 0.f;
    float g = 1.f;
    if (gate && !gate_elems) g = 1.f / (1.f + expf(-to_f32(gate[r * ldg + h])));
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        const float o = maps > 1 ? to_f32(a1[c]) - l * to_f32(a1[dv + c]) : to_f32(a1[c]);
        ss += o * o;
    }
    float inv = 1.f;
    if (norm) {
        ss = block_sum(ss, red);
        inv = 1.f / sqrtf(ss / (float)dv + eps);
    }
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        const float o = maps > 1 ? to_f32(a1[c]) - l * to_f32(a1[dv + c]) : to_f32(a1[c]);
        if (gate && gate_elems) g = 1.f / (1.f + expf(-to_f32(gate[r * ldg + (size_t)h * dv + c])));
        out[r * ld_out + (size_t)h * dv + c] = from_f32<T>(o * inv * mul * g);
    }
}

extern "C" int gi_attn_finish(const void* att, int att_dtype, int maps, const float* lam, float eps, int norm, float mul,
                              const void* gate, long long ldg, void* out, long long ld_out, int act_dtype, int n_rows,
                              int heads, int dv, int gate_elems, void* stream) {
    GI_REQUIRE(n_rows >= 0 && heads > 0 && heads <= 65535 && dv > 0 && (maps == 1 || maps == 2),
               "gi_attn_finish: %d heads of %d values in %d maps", heads, dv, maps);
    GI_REQUIRE(maps == 1 || lam, "gi_attn_finish: two maps need their factor");
    GI_REQUIRE(ld_out >= (long long)heads * dv, "gi_attn_finish: output rows shorter than the heads");
    if (n_rows == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = dv > 128 ? 128 : (dv > 64 ? 64 : 32);
    dim3 grid(n_rows, heads);
    if (att_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_F32)
        gi_launch(attn_finish_kernel<float, float>, grid, dim3(threads), 0, s, (const float*)att, maps, lam, eps, norm, mul,
                  (const float*)gate, ldg, (float*)out, ld_out, heads, dv, gate_elems);
    else if (att_dtype == GI_DTYPE_F32 && act_dtype == GI_DTYPE_BF16)
        gi_launch(attn_finish_kernel<float, bf16>, grid, dim3(threads), 0, s, (const float*)att, maps, lam, eps, norm, mul,
                  (const bf16*)gate, ldg, (bf16*)out, ld_out, heads, dv, gate_elems);
    else if (att_dtype == GI_DTYPE_BF16 && act_dtype == GI_DTYPE_BF16)
        gi_launch(attn_finish_kernel<bf16, bf16>, grid, dim3(threads), 0, s, (const bf16*)att, maps, lam, eps, norm, mul,
                  (const bf16*)gate, ldg, (bf16*)out, ld_out, heads, dv, gate_elems);
    else
        GI_REQUIRE(false, "gi_attn_finish: attention dtype %d with activation dtype %d", att_dtype, act_dtype);
    return gi_check_launch("gi_attn_finish");
}
