// A matrix memory with exponential gates (the mLSTM cell of xLSTM), per head, float32 state:
//
//   i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap))         log gates, one of each per head
//   m_t = max(f + m_(t-1), i)                                                          from 0 before the first token
//   S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,   n_t the same with k alone;  both from 0
//   o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)            q the projection times key_dim^-1/2
//
// A block owns one (sequence, head, slice of 32 value columns) and walks the sequence's tokens of the step in order,
// so prompts, portions and single tokens give the same bits.  All its warps but one walk S like the other scans, with
// two value columns to a thread and products and sums in pairs (general_delta.cu says why).  One
// more warp keeps n (its keys spread over the lanes), makes the denominators' reciprocals, and makes the NEXT chunk's gates while
// the others walk: a lane takes a token's tanh, logarithm and exponentials, and the running maximum goes through the
// lanes in order.  The output is divided once per chunk.  Every slice of a head has a copy of n and m of its
// own in the state row, because no order is known between the blocks that read and write them.
// State row: per head [value column][key, padded] as the other scans, then a padded n per slice, then an m per slice.
// NikolayBlagoev/garlic-inference has no recurrent mixer.
#include "scan.cuh"

#define MM_DEN_EPS 1e-6f
#define MM_TC(DP) ((DP) <= 32 || (DP) > 128 ? 16 : 32)              // tokens in shared memory at a time

static __host__ __device__ __forceinline__ long long mm_head_floats(int DP, int dv) {
    const int ns = (dv + SCAN_VS - 1) / SCAN_VS;
    return (long long)dv * DP + (long long)ns * DP + (ns + 3) / 4 * 4;
}

template <typename T, int R, int P>
__global__ void __launch_bounds__(SCAN_HALF * P + 32)
matrix_memory_scan_kernel(const T* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                          const float* __restrict__ gates, long long ldg, int i_off, int f_off,
                          const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap, float q_scale,
                          float* __restrict__ state, long long state_stride, const int* __restrict__ spans,
                          const int* __restrict__ tok_slot, float* __restrict__ out, int H, int d, int dv, int vec) {
    gi_pdl_start();
    constexpr int DP = R * P;
    constexpr int TC = MM_TC(DP);
    constexpr int WALKERS = SCAN_HALF * P, WARPS = WALKERS / 32;     // threads and warps that walk S
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
    const int part = threadIdx.x % P, vl = walker ? threadIdx.x / P : 0;        // columns vl and vl + SCAN_HALF of the slice
    const bool live_a = walker && v0 + vl < dv, live_b = walker && v0 + vl + SCAN_HALF < dv;
    if (slot < 0) {
        for (int i = threadIdx.x; i < len * SCAN_VS; i += blockDim.x)
            if (v0 + i % SCAN_VS < dv) out[(size_t)(start + i / SCAN_VS) * H * dv + h * dv + v0 + i % SCAN_VS] = 0.f;
        return;
    }
    float* head = state + (size_t)slot * state_stride + (size_t)h * mm_head_floats(DP, dv);
    float* st = head + (size_t)v0 * DP;
    float* n_st = head + (size_t)dv * DP + (size_t)slice * DP;
    float* m_st = head + (size_t)dv * DP + (size_t)gridDim.z * DP + slice;
    constexpr int NN = (DP + 31) / 32;                     // keys of n per lane of the last warp: lane, lane + 32, ...
    f32x2 Sa[R / 2], Sb[R / 2];
    float n_reg[NN];
    scan_load_pairs<R, P>(Sa, st + (size_t)vl * DP, part, live_a);
    scan_load_pairs<R, P>(Sb, st + (size_t)(vl + SCAN_HALF) * DP, part, live_b);
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
#pragma unroll
        for (int t = 0; t < TC; ++t) {                     // the running maximum, token after token
            const float ft = __shfl_sync(0xffffffffu, f, t), it = __shfl_sync(0xffffffffu, i, t);
            const float m_new = fmaxf(ft + m_run, it);
            if (t == lane) { m_before = m_run; m_mine = m_new; }
            m_run = t < tc ? m_new : m_run;
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
    uint32_t pv[TPW];
    // (no branches around the loads: general_delta.cu says why)
    const int vc = min(v0 + lane, dv - 1);
    auto fetch = [&](int t0) {
        const int last = min(TC, len - t0) - 1;
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const T* row = qkv + (size_t)(start + t0 + min(warp + WARPS * i, last)) * ld;
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                const int c = h * d + min((lane + 32 * n) * 4, d - 4);
                raw4_load(pq[i][n], row + q_off + c);
                raw4_load(pk[i][n], row + k_off + c);
            }
            pv[i] = raw1_load(row + v_off + h * dv + vc);
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
                if (vec) {                                 // rows behind the chunk's last get what is not read
#pragma unroll
                    for (int n = 0; n < NQ; ++n) {
                        const int c = (lane + 32 * n) * 4;
                        if (c >= DP) continue;
                        raw_arrived(pq[i][n]); raw_arrived(pk[i][n]);
                        float4 q4 = raw4_f32(pq[i][n]), k4 = raw4_f32(pk[i][n]);
                        if (c >= d) { raw4_zero(q4); raw4_zero(k4); }      // d is a multiple of 4 here
                        *reinterpret_cast<float4*>(&q_s[t][c]) = make_float4(q4.x * q_scale, q4.y * q_scale, q4.z * q_scale, q4.w * q_scale);
                        *reinterpret_cast<float4*>(&k_s[t][c]) = k4;
                    }
                    raw_arrived(pv[i]);
                    v_s[t][lane] = raw1_f32<T>(pv[i]);
                } else if (t < tc) {
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
            auto token = [&](int t, float& oa, float& ob) {        // the state, and this lane's parts of the read-out
                const float put = put_s[buf][t];
                const f32x2 keep = both2(keep_s[buf][t]), wa = both2(put * v_s[t][vl]), wb = both2(put * v_s[t][vl + SCAN_HALF]);
                f32x2 oa0 = 0ull, oa1 = 0ull, ob0 = 0ull, ob1 = 0ull;
#pragma unroll
                for (int i = 0; i < R / 4; ++i) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(&k_s[t][KEY_OF(i, part)]);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(&q_s[t][KEY_OF(i, part)]);
                    Sa[2 * i] = fma2(keep, Sa[2 * i], mul2(kk.x, wa));          oa0 = fma2(Sa[2 * i], qq.x, oa0);
                    Sa[2 * i + 1] = fma2(keep, Sa[2 * i + 1], mul2(kk.y, wa));  oa1 = fma2(Sa[2 * i + 1], qq.y, oa1);
                    Sb[2 * i] = fma2(keep, Sb[2 * i], mul2(kk.x, wb));          ob0 = fma2(Sb[2 * i], qq.x, ob0);
                    Sb[2 * i + 1] = fma2(keep, Sb[2 * i + 1], mul2(kk.y, wb));  ob1 = fma2(Sb[2 * i + 1], qq.y, ob1);
                }
                oa = sum2(oa0, oa1);
                ob = sum2(ob0, ob1);
            };
            int t = 0;
            for (; t + P <= tc; t += P) {
                float oa[P], ob[P];
#pragma unroll
                for (int u = 0; u < P; ++u) token(t + u, oa[u], ob[u]);
                o_s[t + part][vl] = part_sum_tokens<P>(oa, part);
                o_s[t + part][vl + SCAN_HALF] = part_sum_tokens<P>(ob, part);
            }
            for (; t < tc; ++t) {
                float oa, ob;
                token(t, oa, ob);
                oa = part_sum<P>(oa);
                ob = part_sum<P>(ob);
                if (part == 0) { o_s[t][vl] = oa; o_s[t][vl + SCAN_HALF] = ob; }
            }
        } else {
            if (more) fetch_gates(t0 + TC);
            auto key_sums = [&](int t) {                   // one token: n, and this lane's part of n . q
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
                return dot;
            };
            int t = 0;
            for (; t + 8 <= tc; t += 8) {                  // eight tokens' sums over the lanes side by side
                float dot[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) dot[u] = key_sums(t + u);
                float mine = part_sum_tokens<8>(dot, lane & 7);
                mine += __shfl_xor_sync(0xffffffffu, mine, 8);
                mine += __shfl_xor_sync(0xffffffffu, mine, 16);
                if (lane < 8) den_s[t + lane] = 1.f / (fmaxf(fabsf(mine), floor_s[buf][t + lane]) + MM_DEN_EPS);
            }
            for (; t < tc; ++t) {
                const float dot = part_sum<32>(key_sums(t));
                if (lane == 0) den_s[t] = 1.f / (fmaxf(fabsf(dot), floor_s[buf][t]) + MM_DEN_EPS);
            }
            if (more) make_gates(t0 + TC, buf ^ 1);
        }
        __syncthreads();
        if (walker) {
            float* o_row = out + (size_t)(start + t0 + warp) * H * dv + h * dv + v0 + lane;
#pragma unroll
            for (int i = 0; i < TPW; ++i) {
                const int t = warp + WARPS * i;
                if (t < tc && v0 + lane < dv) o_row[(size_t)i * WARPS * H * dv] = o_s[t][lane] * den_s[t];
            }
        }
    }
    if (live_a) scan_store_pairs<R, P>(Sa, st + (size_t)vl * DP, part);
    if (live_b) scan_store_pairs<R, P>(Sb, st + (size_t)(vl + SCAN_HALF) * DP, part);
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
    gi_launch(matrix_memory_scan_kernel<T, R, P>, grid, dim3(SCAN_HALF * P + 32), 0, s, (const T*)qkv, ld, q_off, k_off, \
              v_off, gates, ldg, i_off, f_off, i_bias, f_bias, cap, q_scale, state, state_stride, spans, tok_slot, out,  \
              H, d, dv, vec)
    if (act_dtype == GI_DTYPE_F32) SCAN_SIZES(MM_LAUNCH, float)
    else if (act_dtype == GI_DTYPE_BF16) SCAN_SIZES(MM_LAUNCH, bf16)
    else GI_REQUIRE(false, "gi_matrix_memory_scan: activation dtype %d", act_dtype);
#undef MM_LAUNCH
    return gi_check_launch("gi_matrix_memory_scan");
}
