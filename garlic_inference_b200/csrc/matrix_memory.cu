// A matrix memory with exponential gates (the mLSTM cell of xLSTM), per head, float32 state:
//
//   i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap))         log gates, one of each per head
//   m_t = max(f + m_(t-1), i)                                                          from 0 before the first token
//   S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,   n_t the same with k alone;  both from 0
//   o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)            q the projection times key_dim^-1/2
//
// A block owns one (sequence, head, slice of 32 value columns) and walks the sequence's tokens of the step in order,
// so prompts, portions and single tokens give the same bits.  Its first P warps walk S like the other scans.  One
// more warp keeps n (its keys spread over the lanes), makes the denominators, and makes the NEXT chunk's gates while
// the others walk: a lane takes a token's tanh, logarithm and exponentials, and the running maximum goes through the
// lanes in order.  The output's division happens once per chunk.  Every slice of a head has a copy of n and m of its
// own in the state row, because no order is known between the blocks that read and write them.
// State row: per head [value column][key, padded] as the other scans, then a padded n per slice, then an m per slice.
// NikolayBlagoev/garlic-inference has no recurrent mixer.
#include "scan.cuh"

#define MM_DEN_EPS 1e-6f

static __host__ __device__ __forceinline__ long long mm_head_floats(int DP, int dv) {
    const int ns = (dv + SCAN_VS - 1) / SCAN_VS;
    return (long long)dv * DP + (long long)ns * DP + (ns + 3) / 4 * 4;
}

template <typename T, int R, int P>
__global__ void __launch_bounds__(SCAN_VS * P + 32)
matrix_memory_scan_kernel(const T* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                          const float* __restrict__ gates, long long ldg, int i_off, int f_off,
                          const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap, float q_scale,
                          float* __restrict__ state, long long state_stride, const int* __restrict__ spans,
                          const int* __restrict__ tok_slot, float* __restrict__ out, int H, int d, int dv, int vec) {
    gi_pdl_start();
    constexpr int DP = R * P;
    constexpr int TC = SCAN_TC(DP);
    constexpr int WALKERS = SCAN_VS * P, WARPS = P;        // threads and warps that walk S
    __shared__ __align__(16) float q_s[TC][DP];
    __shared__ __align__(16) float k_s[TC][DP];
    __shared__ float v_s[TC][SCAN_VS];
    __shared__ __align__(16) float o_s[TC][SCAN_O_LD];
    __shared__ float keep_s[2][32], put_s[2][32], floor_s[2][32], den_s[32];
    int slot, start, len;
    scan_span(spans, tok_slot, blockIdx.x, slot, start, len);
    const int h = blockIdx.y, slice = blockIdx.z, v0 = slice * SCAN_VS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const bool walker = warp < WARPS;
    const int part = threadIdx.x % P, vl = walker ? threadIdx.x / P : 0, v = v0 + vl;
    const bool live = walker && v < dv;
    if (slot < 0) {
        for (int t = 0; t < len; ++t)
            if (live && part == 0) out[(size_t)(start + t) * H * dv + h * dv + v] = 0.f;
        return;
    }
    float* head = state + (size_t)slot * state_stride + (size_t)h * mm_head_floats(DP, dv);
    float* st = head + (size_t)(live ? v : 0) * DP;
    float* n_st = head + (size_t)dv * DP + (size_t)slice * DP;
    float* m_st = head + (size_t)dv * DP + (size_t)gridDim.z * DP + slice;
    constexpr int NN = (DP + 31) / 32;                     // keys of n per lane of the last warp: lane, lane + 32, ...
    float S[R], n_reg[NN];
    if (live) scan_load_state<R, P>(S, st, part);
    else {
#pragma unroll
        for (int e = 0; e < R; ++e) S[e] = 0.f;
    }
    float m_run = 0.f, zi = 0.f, zf = 0.f;
    if (!walker) {
#pragma unroll
        for (int e = 0; e < NN; ++e) n_reg[e] = lane + 32 * e < DP ? n_st[lane + 32 * e] : 0.f;
        m_run = *m_st;
    }
    const float bi = i_bias[h], bf = f_bias[h];
    auto fetch_gates = [&](int t0) {                       // lane t: the logits of token t0 + t
        if (lane < min(TC, len - t0)) {
            const float* g = gates + (size_t)(start + t0 + lane) * ldg;
            zi = g[i_off + h];
            zf = g[f_off + h];
        }
    };
    auto make_gates = [&](int t0, int buf) {
        const int tc = min(TC, len - t0);
        const float i = cap * tanhf((zi + bi) / cap);
        const float zc = cap * tanhf((zf + bf) / cap);
        const float f = fminf(zc, 0.f) - log1pf(expf(-fabsf(zc)));
        float m_before = 0.f, m_mine = 0.f;
        for (int t = 0; t < tc; ++t) {                     // the running maximum, token after token
            const float ft = __shfl_sync(0xffffffffu, f, t), it = __shfl_sync(0xffffffffu, i, t);
            const float m_new = fmaxf(ft + m_run, it);
            if (t == lane) { m_before = m_run; m_mine = m_new; }
            m_run = m_new;
        }
        if (lane < tc) {
            keep_s[buf][lane] = expf(f + m_before - m_mine);
            put_s[buf][lane] = expf(i - m_mine);
            floor_s[buf][lane] = expf(-m_mine);
        }
    };
    // staging: warp w takes tokens w, w + WARPS, ... of a chunk; the next chunk's raw values are asked for before this
    // chunk is walked
    typedef typename Raw4<T>::type raw_t;
    constexpr int TPW = (TC + WARPS - 1) / WARPS;
    constexpr int NQ = (DP / 4 + 31) / 32;
    raw_t pq[TPW][NQ], pk[TPW][NQ];
    float pv[TPW];
    auto fetch = [&](int t0) {
        const int tc = min(TC, len - t0);
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = warp + WARPS * i;
            if (t >= tc) continue;
            const T* row = qkv + (size_t)(start + t0 + t) * ld;
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                const int c = (lane + 32 * n) * 4;
                raw4_zero(pq[i][n]); raw4_zero(pk[i][n]);
                if (c < d) {
                    pq[i][n] = *reinterpret_cast<const raw_t*>(row + q_off + h * d + c);
                    pk[i][n] = *reinterpret_cast<const raw_t*>(row + k_off + h * d + c);
                }
            }
            pv[i] = v0 + lane < dv ? to_f32(row[v_off + h * dv + v0 + lane]) : 0.f;
        }
    };
    if (walker) { if (vec) fetch(0); }
    else { fetch_gates(0); make_gates(0, 0); }
    int buf = 0;
    for (int t0 = 0; t0 < len; t0 += TC, buf ^= 1) {
        const int tc = min(TC, len - t0);
        __syncthreads();                                   // the last chunk's outputs and inputs are done with
        if (walker) {
#pragma unroll
            for (int i = 0; i < TPW; ++i) {
                const int t = warp + WARPS * i;
                if (t >= tc) continue;
                if (vec) {
#pragma unroll
                    for (int n = 0; n < NQ; ++n) {
                        const int c = (lane + 32 * n) * 4;
                        if (c >= DP) continue;
                        const float4 q4 = raw4_f32(pq[i][n]);
                        *reinterpret_cast<float4*>(&q_s[t][c]) = make_float4(q4.x * q_scale, q4.y * q_scale, q4.z * q_scale, q4.w * q_scale);
                        *reinterpret_cast<float4*>(&k_s[t][c]) = raw4_f32(pk[i][n]);
                    }
                    v_s[t][lane] = pv[i];
                } else {
                    const T* row = qkv + (size_t)(start + t0 + t) * ld;
                    for (int c = lane; c < DP; c += 32) {
                        q_s[t][c] = c < d ? to_f32(row[q_off + h * d + c]) * q_scale : 0.f;
                        k_s[t][c] = c < d ? to_f32(row[k_off + h * d + c]) : 0.f;
                    }
                    v_s[t][lane] = v0 + lane < dv ? to_f32(row[v_off + h * dv + v0 + lane]) : 0.f;
                }
            }
        }
        __syncthreads();
        const bool more = t0 + TC < len;
        if (walker) {
            if (vec && more) fetch(t0 + TC);
            auto token = [&](int t) {                      // one token: the state, and this lane's part of the read-out
                const float keep = keep_s[buf][t], w = put_s[buf][t] * v_s[t][vl];
                float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
                for (int i = 0; i < R / 4; ++i) {
                    const float4 kk = *reinterpret_cast<const float4*>(&k_s[t][KEY_OF(i, part)]);
                    const float4 qq = *reinterpret_cast<const float4*>(&q_s[t][KEY_OF(i, part)]);
                    S[4 * i] = fmaf(keep, S[4 * i], kk.x * w);          o0 = fmaf(S[4 * i], qq.x, o0);
                    S[4 * i + 1] = fmaf(keep, S[4 * i + 1], kk.y * w);  o1 = fmaf(S[4 * i + 1], qq.y, o1);
                    S[4 * i + 2] = fmaf(keep, S[4 * i + 2], kk.z * w);  o2 = fmaf(S[4 * i + 2], qq.z, o2);
                    S[4 * i + 3] = fmaf(keep, S[4 * i + 3], kk.w * w);  o3 = fmaf(S[4 * i + 3], qq.w, o3);
                }
                return (o0 + o1) + (o2 + o3);
            };
            int t = 0;
            for (; t + P <= tc; t += P) {
                float o[P];
#pragma unroll
                for (int u = 0; u < P; ++u) o[u] = token(t + u);
                o_s[t + part][vl] = part_sum_tokens<P>(o, part);
            }
            for (; t < tc; ++t) {
                const float o = part_sum<P>(token(t));
                if (part == 0) o_s[t][vl] = o;
            }
        } else {
            if (more) fetch_gates(t0 + TC);
            for (int t = 0; t < tc; ++t) {
                const float keep = keep_s[buf][t], put = put_s[buf][t];
                float dot = 0.f;
#pragma unroll
                for (int e = 0; e < NN; ++e) {
                    const int c = lane + 32 * e;
                    if (c < DP) {
                        n_reg[e] = fmaf(keep, n_reg[e], put * k_s[t][c]);
                        dot = fmaf(n_reg[e], q_s[t][c], dot);
                    }
                }
                dot = warp_sum(dot);
                if (lane == 0) den_s[t] = fmaxf(fabsf(dot), floor_s[buf][t]) + MM_DEN_EPS;
            }
            if (more) make_gates(t0 + TC, buf ^ 1);
        }
        __syncthreads();
        if (walker)
            for (int i = threadIdx.x; i < tc * SCAN_VS; i += WALKERS) {
                const int t = i / SCAN_VS, c = i - t * SCAN_VS;
                if (v0 + c < dv) out[(size_t)(start + t0 + t) * H * dv + h * dv + v0 + c] = o_s[t][c] / den_s[t];
            }
    }
    if (live) scan_store_state<R, P>(S, st, part);
    if (!walker) {
#pragma unroll
        for (int e = 0; e < NN; ++e)
            if (lane + 32 * e < DP) n_st[lane + 32 * e] = n_reg[e];
        if (lane == 0) *m_st = m_run;
    }
}

// Floats of one head's state row for key dimension d and value dimension dv (-1: a key dimension beyond 256).
extern "C" long long gi_matrix_memory_state_floats(int d, int dv) {
    const int DP = scan_padded(d);
    return DP && dv > 0 ? mm_head_floats(DP, dv) : -1;
}

// qkv: T [n, ld], q of head h at column q_off + h d, k at k_off + h d, v at v_off + h dv.  gates: float32 [n, ldg], the
// logits of head h at i_off + h and f_off + h; i_bias, f_bias float32 [H].  out float32 [n, H dv].
extern "C" int gi_matrix_memory_scan(const void* qkv, long long ld, int act_dtype, int q_off, int k_off, int v_off,
                                     const float* gates, long long ldg, int i_off, int f_off, const float* i_bias,
                                     const float* f_bias, float cap, float q_scale, float* state, long long state_stride,
                                     const int* spans, const int* tok_slot, float* out, int n_seq, int H, int d, int dv,
                                     void* stream) {
    const int DP = scan_padded(d);
    GI_REQUIRE(n_seq >= 0 && H > 0 && d > 0 && dv > 0 && DP > 0, "gi_matrix_memory_scan: key dimension %d (at most 256)", d);
    GI_REQUIRE(H <= 65535 && (dv + SCAN_VS - 1) / SCAN_VS <= 65535, "gi_matrix_memory_scan: %d heads of %d values", H, dv);
    GI_REQUIRE(cap > 0.f, "gi_matrix_memory_scan: a gate cap of %f", (double)cap);
    GI_REQUIRE(state_stride >= H * mm_head_floats(DP, dv) && state_stride % 4 == 0, "gi_matrix_memory_scan: state rows of "
               "%lld floats are shorter than %lld or no multiple of 4", state_stride, H * mm_head_floats(DP, dv));
    if (n_seq == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(n_seq, H, (dv + SCAN_VS - 1) / SCAN_VS);
    const int esz = act_dtype == GI_DTYPE_F32 ? 4 : 2;
    const int vec = d % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && (uintptr_t)qkv % (4 * esz) == 0;
#define MM_LAUNCH(T, R, P)                                                                                            \
    gi_launch(matrix_memory_scan_kernel<T, R, P>, grid, dim3(SCAN_VS * P + 32), 0, s, (const T*)qkv, ld, q_off, k_off, \
              v_off, gates, ldg, i_off, f_off, i_bias, f_bias, cap, q_scale, state, state_stride, spans, tok_slot, out,  \
              H, d, dv, vec)
#define MM_DISPATCH(T)                                                                                                \
    switch (DP) {                                                                                                     \
        case 16: MM_LAUNCH(T, 4, 4); break;                                                                           \
        case 32: MM_LAUNCH(T, 8, 4); break;                                                                           \
        case 64: MM_LAUNCH(T, 8, 8); break;                                                                           \
        case 128: MM_LAUNCH(T, 16, 8); break;                                                                         \
        default: MM_LAUNCH(T, 32, 8); break;                                                                          \
    }
    if (act_dtype == GI_DTYPE_F32) MM_DISPATCH(float)
    else if (act_dtype == GI_DTYPE_BF16) MM_DISPATCH(bf16)
    else GI_REQUIRE(false, "gi_matrix_memory_scan: activation dtype %d", act_dtype);
#undef MM_DISPATCH
#undef MM_LAUNCH
    return gi_check_launch("gi_matrix_memory_scan");
}
