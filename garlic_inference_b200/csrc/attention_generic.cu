// Attention over the paged cache for any number of new tokens per sequence,
// float32 or bfloat16, any head_dim up to 1024.
//
// This is the engine's exact path: the float32 engine uses it for prompts and
// for decoding alike, and the bfloat16 engine uses it for head sizes its
// tensor-core kernels do not take.  One block computes one (token, query
// head).  Keys are visited in chunks of 32 aligned to absolute positions
// (chunk c = keys 32c..32c+31), chunk c by warp c mod 4, and the four partial
// results are merged in warp order: the result at a position therefore does
// not depend on how the tokens were cut into steps, on the batch, or on where
// the pages lie.
//
//   o = softmax_j( q . k_j * scale ) v_j   over keys j <= pos, and j > pos - window
//                                           when window > 0
// With `sinks` (one number per query head) the softmax's denominator also holds exp(sink_h): a key without a
// value, not scaled, counted once.  With d_v < d only the first d_v columns of a value row are summed and the
// output rows are d_v wide (a cache whose rows serve as keys in full and as values in part).
// Query head h reads key/value head h / (n_q / n_kv).  Scores, softmax and the
// weighted sum are float32.
// Three more parameters, for mixers beside plain grouped-query attention:
//   chunk > 0    a query at position i sees only the keys j <= i of its own chunk, floor(j / chunk) = floor(i / chunk)
//                (chunks are counted from position 0 of the sequence);
//   values of their own shape: the value pool has n_vh heads per page with rows of v_row elements, which may be
//                wider or narrower than a key row;
//   maps > 1     every head owns `maps` softmaxes over the same values (the maps of a differential attention):
//                the n_q query rows of a token are laid out [head][map], the n_kv key heads [key head][map], and
//                row h = head * maps + map reads key head (head / group) * maps + map and value head head / group,
//                group = (n_q / maps) / n_vh;
//   dist_bias    a learned bias per distance and query row, float32 [n_dist, n_q]: the score of key j for the query at
//                position i gets dist_bias[min(i - j, n_dist - 1), row] added after the scaling;
//   means        beside the keys of its window a query sees one more row (key and value) for every block of `block`
//                positions that lies wholly before the window, block b from b block + block - 1 <= i - window on; they
//                come from pools of their own and share the softmax (a window is required then).  They are visited
//                before the window's keys, 32 at a time like those;
//   keep_first   the first `keep_first` positions of a sequence stay in sight of every later query beside the window (a
//                window is required); like block rows they are visited before the window's keys, 32 at a time;
//   out_f32      the result is written as float32 whatever the activation type is (a later kernel combines maps).  Upstream hands this to a library
// (src/src-cuda/attention/fattn.cu:74-86: scale 1/sqrt(head_dim), causal mask
// aligned to the last key, float32 intermediates).
#include "common.cuh"
#include <math.h>

#define AG_WARPS 4

// Rows that stand for whole blocks of positions: row b of a sequence in page b / rows of its row of `table`, at row
// b % rows; pools [pages, heads, rows, width].  block = 0: none.
struct BlockRows {
    const void *k, *v;
    const int* table;
    int block, rows, max_pages, n_pages;
};

template <typename T> struct Vec;
template <> struct Vec<float> { static constexpr int N = 4; typedef float4 type; };
template <> struct Vec<bf16> { static constexpr int N = 8; typedef uint4 type; };

__device__ __forceinline__ float dot_vec(const float4& k, const float* q) {
    return k.x * q[0] + k.y * q[1] + k.z * q[2] + k.w * q[3];
}
__device__ __forceinline__ float dot_vec(const uint4& k, const float* q) {
    const __nv_bfloat162* k2 = reinterpret_cast<const __nv_bfloat162*>(&k);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(k2[i]);
        s += f.x * q[2 * i] + f.y * q[2 * i + 1];
    }
    return s;
}

template <typename T, int DPL>
__global__ void __launch_bounds__(AG_WARPS * 32)
attn_generic_kernel(const T* __restrict__ q, const T* __restrict__ k_pool, const T* __restrict__ v_pool,
                    const int* __restrict__ block_table, const int* __restrict__ tok_pos,
                    const int* __restrict__ tok_slot, T* __restrict__ out, int n_q, int n_kv, int d,
                    int page_size, int max_pages, int n_pool_pages, int window, float scale,
                    const void* __restrict__ sinks, int sink_dtype, int d_v, int* __restrict__ status,
                    int chunk, int n_vh, int v_row, int maps, float* __restrict__ out_f32,
                    const float* __restrict__ dist_bias, int n_dist, BlockRows means, int keep_first) {
    gi_pdl_start();
    extern __shared__ float smem[];
    const int dw = d > d_v ? d : d_v;        // width of an accumulator row
    float* q_s = smem;                       // d
    float* acc_s = smem + d;                 // AG_WARPS * dw
    float* m_s = acc_s + AG_WARPS * dw;      // AG_WARPS
    float* l_s = m_s + AG_WARPS;             // AG_WARPS

    const int t = blockIdx.x, h = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    T* o = out ? out + ((size_t)t * n_q + h) * d_v : nullptr;
    float* of = out_f32 ? out_f32 + ((size_t)t * n_q + h) * d_v : nullptr;
    const int slot = tok_slot[t];
    const int pos = tok_pos[t];
    if (slot < 0 || pos < 0 || pos / page_size >= max_pages) {
        for (int i = threadIdx.x; i < d_v; i += blockDim.x) {
            if (of) of[i] = 0.f; else o[i] = from_f32<T>(0.f);
        }
        if (slot >= 0 && threadIdx.x == 0) atomicExch(status, 4);
        return;
    }
    const int head = h / maps, group = (n_q / maps) / n_vh;
    const int kvh = (head / group) * maps + (h - head * maps);
    const int vh = head / group;
    const T* qrow = q + ((size_t)t * n_q + h) * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) q_s[i] = to_f32(qrow[i]) * scale;
    __syncthreads();

    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    const int* bt = block_table + (size_t)slot * max_pages;
    float m = -INFINITY, l = 0.f;
    float acc[DPL];
#pragma unroll
    for (int r = 0; r < DPL; ++r) acc[r] = 0.f;

    constexpr int VN = Vec<T>::N;
    typedef typename Vec<T>::type vec_t;
    // blocks the query sees: b with (b + 1) block <= pos - window + 1
    const int n_blocks = means.block > 0 && pos >= window ? (pos - window + 1) / means.block : 0;
    // first tokens that stay in sight: those that the window has left behind
    const int n_kept = window > 0 ? min(keep_first, lo) : 0;
    const int lead_chunks = (max(n_blocks, n_kept) + 31) / 32, first_chunk = lo / 32;
    const int padded = (lead_chunks + AG_WARPS - 1) / AG_WARPS * AG_WARPS;
    const int* mbt = means.block > 0 ? means.table + (size_t)slot * means.max_pages : nullptr;
    // the chunks of blocks (or of kept first tokens), then the chunks of keys: chunk c to warp c mod 4, counted from the
    // first of each kind
    for (int cc = warp; cc < padded + pos / 32 - first_chunk + 1; cc += AG_WARPS) {
        const bool lead = cc < padded, of_blocks = lead && means.block > 0;
        const int c = lead ? cc : cc - padded + first_chunk;
        const int j = c * 32 + lane;
        const bool valid = lead ? j < max(n_blocks, n_kept) : j >= lo && j <= pos;
        long long row = -1;                  // element offset of this lane's key row (-1: none)
        long long vrow = 0;                  // and of its value row
        float s = -INFINITY;
        const T* kp = of_blocks ? (const T*)means.k : k_pool;
        const T* vp = of_blocks ? (const T*)means.v : v_pool;
        if (valid) {
            const int rows = of_blocks ? means.rows : page_size, lp = j / rows;
            const int page = of_blocks ? (lp < means.max_pages ? mbt[lp] : -1) : bt[lp];
            if (page < 0 || page >= (of_blocks ? means.n_pages : n_pool_pages)) {
                atomicExch(status, 5);
            } else {
                row = (((long long)page * n_kv + kvh) * rows + (j - lp * rows)) * d;
                vrow = (((long long)page * n_vh + vh) * rows + (j - lp * rows)) * v_row;
                float a = 0.f;
                if (d % VN == 0) {               // rows start on 16 bytes: vector loads
                    const vec_t* kr = reinterpret_cast<const vec_t*>(kp + row);
                    for (int i = 0; i < d / VN; ++i) a += dot_vec(kr[i], q_s + i * VN);
                } else {
                    for (int i = 0; i < d; ++i) a = fmaf(to_f32(kp[row + i]), q_s[i], a);
                }
                s = dist_bias ? a + dist_bias[(size_t)min(pos - j, n_dist - 1) * n_q + h] : a;
            }
        }
        const float cmax = warp_max(s);
        if (cmax == -INFINITY) continue;
        const float m_new = fmaxf(m, cmax);
        const float corr = expf(m - m_new);              // 0 when m is -inf
        const float p = row >= 0 ? expf(s - m_new) : 0.f;
        l = l * corr + warp_sum(p);
        m = m_new;
#pragma unroll
        for (int r = 0; r < DPL; ++r) acc[r] *= corr;
        for (int jj = 0; jj < 32; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const long long rj = __shfl_sync(0xffffffffu, row, jj);
            const long long vj = __shfl_sync(0xffffffffu, vrow, jj);
            if (rj < 0) continue;
            const T* vr = vp + vj;
#pragma unroll
            for (int r = 0; r < DPL; ++r) {
                const int i = lane + 32 * r;
                if (i < d_v) acc[r] += pj * to_f32(vr[i]);
            }
        }
    }
    if (lane == 0) { m_s[warp] = m; l_s[warp] = l; }
#pragma unroll
    for (int r = 0; r < DPL; ++r) {
        const int i = lane + 32 * r;
        if (i < dw) acc_s[warp * dw + i] = acc[r];
    }
    __syncthreads();
    float M = -INFINITY;
    for (int w = 0; w < AG_WARPS; ++w) M = fmaxf(M, m_s[w]);
    const float sink = sinks ? load_w(sinks, sink_dtype, h) : -INFINITY;
    M = fmaxf(M, sink);
    float L = 0.f;
    for (int w = 0; w < AG_WARPS; ++w) L += (m_s[w] == -INFINITY ? 0.f : expf(m_s[w] - M) * l_s[w]);
    if (sinks) L += expf(sink - M);
    for (int i = threadIdx.x; i < d_v; i += blockDim.x) {
        float v = 0.f;
        for (int w = 0; w < AG_WARPS; ++w)
            if (m_s[w] != -INFINITY) v += expf(m_s[w] - M) * acc_s[w * dw + i];
        const float res = L > 0.f ? v / L : 0.f;
        if (of) of[i] = res; else o[i] = from_f32<T>(res);
    }
}

template <typename T>
static int launch_generic(const void* q, const void* k_pool, const void* v_pool, const int* block_table,
                          const int* tok_pos, const int* tok_slot, void* out, int n_tokens, int n_q, int n_kv,
                          int d, int page_size, int max_pages, int n_pool_pages, int window, float scale,
                          const void* sinks, int sink_dtype, int d_v, int* status, int chunk, int n_vh, int v_row,
                          int maps, float* out_f32, const float* dist_bias, int n_dist, const BlockRows& means,
                          int keep_first, cudaStream_t s) {
    dim3 grid(n_tokens, n_q);
    const int dw = d > d_v ? d : d_v;
    const size_t smem = ((size_t)d + (size_t)dw * AG_WARPS + 2 * AG_WARPS) * sizeof(float);
#define AG_LAUNCH(DPL)                                                                               \
    gi_launch(attn_generic_kernel<T, DPL>, grid, dim3(AG_WARPS * 32), smem, s,                                     \
        (const T*)q, (const T*)k_pool, (const T*)v_pool, block_table, tok_pos, tok_slot, (T*)out,     \
        n_q, n_kv, d, page_size, max_pages, n_pool_pages, window, scale, sinks, sink_dtype, d_v, status, \
        chunk, n_vh, v_row, maps, out_f32, dist_bias, n_dist, means, keep_first)
    if (dw <= 32) AG_LAUNCH(1);
    else if (dw <= 64) AG_LAUNCH(2);
    else if (dw <= 128) AG_LAUNCH(4);
    else if (dw <= 256) AG_LAUNCH(8);
    else if (dw <= 512) AG_LAUNCH(16);
    else AG_LAUNCH(32);
#undef AG_LAUNCH
    return gi_check_launch("gi_attention_generic");
}

// The general entry point: everything the file's head lists.  `out` is written in the activation type unless
// `out_f32` is given.  Key rows whose width is a multiple of 16 bytes are read with vector loads, others
// element by element; value rows may have any width.
extern "C" int gi_attention_masked(const void* q, const void* k_pool, const void* v_pool, int act_dtype,
                                   const int* block_table, const int* tok_pos, const int* tok_slot,
                                   void* out, int n_tokens, int n_q, int n_kv, int d, int page_size,
                                   int max_pages, int n_pool_pages, int window, float scale, const void* sinks,
                                   int sink_dtype, int d_v, int* status, int chunk, int n_vh, int v_row, int maps,
                                   float* out_f32, const float* dist_bias, int n_dist, const void* mean_k,
                                   const void* mean_v, const int* mean_table, int mean_block, int mean_rows,
                                   int mean_max_pages, int mean_pages, int keep_first, void* stream) {
    GI_REQUIRE(keep_first >= 0 && (keep_first == 0 || (window > 0 && chunk == 0 && mean_block == 0)), "gi_attention_generic: "
               "kept first tokens come with a window, without chunks and rows for blocks");
    GI_REQUIRE(n_tokens >= 0 && n_q > 0 && n_kv > 0 && d > 0, "gi_attention_generic: sizes must be positive");
    GI_REQUIRE(!dist_bias || n_dist > 0, "gi_attention_generic: a distance bias of %d rows", n_dist);
    GI_REQUIRE(maps >= 1 && n_vh >= 1 && n_q % maps == 0 && n_kv == n_vh * maps && (n_q / maps) % n_vh == 0,
               "gi_attention_generic: %d query rows and %d key heads in %d maps over %d value heads", n_q, n_kv, maps, n_vh);
    GI_REQUIRE(d <= 1024, "gi_attention_generic: head_dim %d is beyond 1024", d);
    GI_REQUIRE((uintptr_t)k_pool % 16 == 0, "gi_attention_generic: the key pool must start on 16 bytes");
    GI_REQUIRE(n_q <= 65535, "gi_attention_generic: %d query heads is beyond 65535", n_q);
    GI_REQUIRE(d_v > 0 && d_v <= v_row && d_v <= 1024, "gi_attention_generic: %d value columns of rows of %d", d_v, v_row);
    GI_REQUIRE(page_size > 0 && max_pages > 0 && window >= 0 && chunk >= 0, "gi_attention_generic: page size, table width, window and chunk");
    GI_REQUIRE(out || out_f32, "gi_attention_generic: no output");
    GI_REQUIRE(mean_block == 0 || (mean_block > 0 && window > 0 && chunk == 0 && !dist_bias && mean_rows > 0 && mean_max_pages > 0 &&
               mean_pages > 0 && (uintptr_t)mean_k % 16 == 0), "gi_attention_generic: rows for blocks of %d positions come with a window, "
               "without chunks and distance biases", mean_block);
    const BlockRows means = {mean_k, mean_v, mean_table, mean_block, mean_rows, mean_max_pages, mean_pages};
    if (n_tokens == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == GI_DTYPE_F32)
        return launch_generic<float>(q, k_pool, v_pool, block_table, tok_pos, tok_slot, out, n_tokens, n_q, n_kv, d,
                                     page_size, max_pages, n_pool_pages, window, scale, sinks, sink_dtype, d_v, status,
                                     chunk, n_vh, v_row, maps, out_f32, dist_bias, n_dist, means, keep_first, s);
    if (act_dtype == GI_DTYPE_BF16)
        return launch_generic<bf16>(q, k_pool, v_pool, block_table, tok_pos, tok_slot, out, n_tokens, n_q, n_kv, d,
                                    page_size, max_pages, n_pool_pages, window, scale, sinks, sink_dtype, d_v, status,
                                    chunk, n_vh, v_row, maps, out_f32, dist_bias, n_dist, means, keep_first, s);
    GI_REQUIRE(false, "gi_attention_generic: activation dtype %d", act_dtype);
}

// Plain grouped-query attention: keys and values of one shape, one softmax per head, no chunks.
extern "C" int gi_attention_generic(const void* q, const void* k_pool, const void* v_pool, int act_dtype,
                                    const int* block_table, const int* tok_pos, const int* tok_slot,
                                    void* out, int n_tokens, int n_q, int n_kv, int d, int page_size,
                                    int max_pages, int n_pool_pages, int window, float scale, const void* sinks,
                                    int sink_dtype, int d_v, int* status, void* stream) {
    GI_REQUIRE(d_v > 0 && d_v <= d, "gi_attention_generic: %d value columns of rows of %d", d_v, d);
    return gi_attention_masked(q, k_pool, v_pool, act_dtype, block_table, tok_pos, tok_slot, out, n_tokens, n_q, n_kv, d,
                               page_size, max_pages, n_pool_pages, window, scale, sinks, sink_dtype, d_v, status, 0, n_kv, d,
                               1, nullptr, nullptr, 0, nullptr, nullptr, nullptr, 0, 0, 0, 0, 0, stream);
}
