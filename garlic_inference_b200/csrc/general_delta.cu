// The generalized delta rule: a decay and a removal rate per head and key channel, float32 state per head.
//
//   w = exp(-exp(-1/2) sigmoid(zw + w0)),   a = sigmoid(za + a0),   u = k / sqrt(|k|^2 + eps)
//   S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T        (the old S in both)
//   o_t = S_t^T r
//
// A block owns one (sequence, head, slice of 32 value columns) and walks the sequence's tokens of the step in order,
// like the other scans, with two value columns to a thread: shared memory hands out 128 bytes a cycle, and what a lane
// reads of a token's keys, decays and rates then serves two columns; products and sums go in pairs.  With y = k^T S_(t-1) of a column and
// z = y / (|k|^2 + eps), channel c of the column becomes w_c S_c + k_c (v - a_c z).  The one sum over the keys that the
// next token waits for is y, so it is started while the present token is written: the loop that renews S also sums
// S against the next token's k.  The read-outs of P tokens are summed over the lanes together.
//   gi_general_delta_rates  w and a in place of their logits, for steps with many tokens: the slices of a head would each
//                           make them again, between two barriers of their walk
//   gi_general_delta_scan   the walk, from logits (a decode step's one token) or from w and a (`ready`); the same bits
// NikolayBlagoev/garlic-inference has no recurrent mixer.
#include "scan.cuh"

#define GD_DECAY 0.60653065971263342f        // exp(-1/2)
#define GD_TC(DP) ((DP) <= 32 || (DP) > 128 ? 8 : 16)              // tokens in shared memory at a time

// Under bfloat16 (FAST) the fast exponential and reciprocal, under float32 the accurate ones.
template <bool FAST> __device__ __forceinline__ float gd_rate(float z) { return FAST ? __fdividef(1.f, 1.f + __expf(-z)) : rc_sigmoid(z); }
template <bool FAST> __device__ __forceinline__ float gd_decay(float z) {
    const float e = -GD_DECAY * gd_rate<FAST>(z);
    return FAST ? __expf(e) : expf(e);
}

template <bool FAST>
__global__ void general_delta_rates_kernel(float* __restrict__ wl, long long ldw, const float* __restrict__ w0,
                                           float* __restrict__ al, long long lda, const float* __restrict__ a0, int n_rows,
                                           int cols) {
    gi_pdl_start();
    const long long total = (long long)n_rows * cols;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / cols;
        const int c = (int)(i - r * cols);
        wl[r * ldw + c] = gd_decay<FAST>(wl[r * ldw + c] + w0[c]);
        al[r * lda + c] = gd_rate<FAST>(al[r * lda + c] + a0[c]);
    }
}
// Four columns at a time, where the rows allow it.
template <bool FAST>
__global__ void general_delta_rates_vec_kernel(float* __restrict__ wl, long long ldw, const float* __restrict__ w0,
                                               float* __restrict__ al, long long lda, const float* __restrict__ a0, int cols) {
    gi_pdl_start();
    for (int c = threadIdx.x * 4; c < cols; c += blockDim.x * 4) {
        float4* w = reinterpret_cast<float4*>(wl + blockIdx.x * ldw + c);
        float4* a = reinterpret_cast<float4*>(al + blockIdx.x * lda + c);
        const float4 zw = *w, za = *a, bw = load4_f32(w0 + c), ba = load4_f32(a0 + c);
        *w = make_float4(gd_decay<FAST>(zw.x + bw.x), gd_decay<FAST>(zw.y + bw.y), gd_decay<FAST>(zw.z + bw.z), gd_decay<FAST>(zw.w + bw.w));
        *a = make_float4(gd_rate<FAST>(za.x + ba.x), gd_rate<FAST>(za.y + ba.y), gd_rate<FAST>(za.z + ba.z), gd_rate<FAST>(za.w + ba.w));
    }
}

extern "C" int gi_general_delta_rates(float* wl, long long ldw, const float* w0, float* al, long long lda, const float* a0,
                                      int act_dtype, int n_rows, int cols, void* stream) {
    GI_REQUIRE(n_rows >= 0 && cols > 0 && ldw >= cols && lda >= cols, "gi_general_delta_rates: sizes");
    if (n_rows == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const bool fast = act_dtype == GI_DTYPE_BF16;
    auto on16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    if (cols % 4 == 0 && ldw % 4 == 0 && lda % 4 == 0 && on16(wl) && on16(al) && on16(w0) && on16(a0)) {
        const int threads = cols >= 1024 ? 256 : 64;
        gi_launch(fast ? general_delta_rates_vec_kernel<true> : general_delta_rates_vec_kernel<false>, dim3(n_rows), dim3(threads), 0, s,
                  wl, ldw, w0, al, lda, a0, cols);
    } else {
        const long long total = (long long)n_rows * cols;
        const int blocks = (int)((total + 255) / 256 > 148 * 16 ? 148 * 16 : (total + 255) / 256);
        gi_launch(fast ? general_delta_rates_kernel<true> : general_delta_rates_kernel<false>, dim3(blocks), dim3(256), 0, s, wl, ldw,
                  w0, al, lda, a0, n_rows, cols);
    }
    return gi_check_launch("gi_general_delta_rates");
}

template <typename T, int R, int P>
__global__ void __launch_bounds__(SCAN_HALF * P)
general_delta_scan_kernel(const T* __restrict__ rkv, long long ld, int r_off, int k_off, int v_off,
                          const float* __restrict__ wl, long long ldw, const float* __restrict__ w0,
                          const float* __restrict__ al, long long lda, const float* __restrict__ a0, float unit_eps,
                          float* __restrict__ state, long long state_stride, const int* __restrict__ spans,
                          const int* __restrict__ tok_slot, float* __restrict__ out, int H, int d, int dv, int vec,
                          int ready) {
    gi_pdl_start();
    constexpr int DP = R * P;
    constexpr int TC = GD_TC(DP);
    constexpr int THREADS = SCAN_HALF * P, WARPS = THREADS / 32;
    __shared__ __align__(16) float r_s[TC][DP];
    __shared__ __align__(16) float k_s[TC][DP];
    __shared__ __align__(16) float w_s[TC][DP];
    __shared__ __align__(16) float a_s[TC][DP];
    __shared__ float v_s[TC][SCAN_VS];
    __shared__ __align__(16) float o_s[TC][SCAN_O_LD];
    __shared__ float inv_s[TC];                            // 1 / (|k|^2 + eps)
    int slot, start, len;
    scan_span(spans, tok_slot, blockIdx.x, slot, start, len);
    const int h = blockIdx.y, v0 = blockIdx.z * SCAN_VS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int part = threadIdx.x % P, vl = threadIdx.x / P;         // columns vl and vl + SCAN_HALF of the slice
    const bool live_a = v0 + vl < dv, live_b = v0 + vl + SCAN_HALF < dv;
    if (slot < 0) {
        for (int i = threadIdx.x; i < len * SCAN_VS; i += THREADS)
            if (v0 + i % SCAN_VS < dv) out[(size_t)(start + i / SCAN_VS) * H * dv + h * dv + v0 + i % SCAN_VS] = 0.f;
        return;
    }
    float* st = state + (size_t)slot * state_stride + ((size_t)h * dv + v0) * DP;
    f32x2 Sa[R / 2], Sb[R / 2];
    scan_load_pairs<R, P>(Sa, st + (size_t)vl * DP, part, live_a);
    scan_load_pairs<R, P>(Sb, st + (size_t)(vl + SCAN_HALF) * DP, part, live_b);
    typedef typename Raw4<T>::type raw_t;
    constexpr int TPW = TC / WARPS;
    constexpr int NQ = (DP / 4 + 31) / 32;
    raw_t pr[TPW][NQ], pk[TPW][NQ];
    float4 pw[TPW][NQ], pa[TPW][NQ];
    uint32_t pv[TPW];
    // Loads without branches around them: a row or a channel beyond the end reads the last one, and what it gave is not
    // used.  Behind a branch each token's loads were waited for before the next token's went out.
    const int vc = min(v0 + lane, dv - 1);
    auto fetch = [&](int t0) {
        const int last = min(TC, len - t0) - 1;
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const size_t at = (size_t)(start + t0 + min(warp + WARPS * i, last));
            const T* row = rkv + at * ld;
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                const int c = h * d + min((lane + 32 * n) * 4, d - 4);
                raw4_load(pr[i][n], row + r_off + c);
                raw4_load(pk[i][n], row + k_off + c);
                raw4_load(pw[i][n], wl + at * ldw + c);
                raw4_load(pa[i][n], al + at * lda + c);
            }
            pv[i] = raw1_load(row + v_off + h * dv + vc);
        }
    };
    float4 bw[NQ], ba[NQ];                                  // the biases of this lane's channels
#pragma unroll
    for (int n = 0; n < NQ; ++n) {
        const int c = (lane + 32 * n) * 4;
        raw4_zero(bw[n]); raw4_zero(ba[n]);
        if (vec && !ready && c < d) {
            bw[n] = *reinterpret_cast<const float4*>(w0 + h * d + c);
            ba[n] = *reinterpret_cast<const float4*>(a0 + h * d + c);
        }
    }
    constexpr bool FAST = sizeof(T) == 2;
    auto sigmoid = [](float z) { return gd_rate<FAST>(z); };
    auto decay = [](float z) { return gd_decay<FAST>(z); };
    if (vec) fetch(0);
    for (int t0 = 0; t0 < len; t0 += TC) {
        const int tc = min(TC, len - t0);
        __syncthreads();                                   // the last chunk's outputs and inputs are done with
        float sk[TPW];
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = warp + WARPS * i;
            sk[i] = 0.f;
            if (vec) {                                     // rows behind the chunk's last get what is not read
#pragma unroll
                for (int n = 0; n < NQ; ++n) {
                    const int c = (lane + 32 * n) * 4;
                    if (c >= DP) continue;
                    raw_arrived(pr[i][n]); raw_arrived(pk[i][n]); raw_arrived(pw[i][n]); raw_arrived(pa[i][n]);
                    const bool in = c < d;             // d is a multiple of 4 here; channels behind it stay zero
                    float4 k4 = raw4_f32(pk[i][n]), r4 = raw4_f32(pr[i][n]);
                    if (!in) { raw4_zero(k4); raw4_zero(r4); }
                    const float4 zw = pw[i][n], za = pa[i][n];
                    *reinterpret_cast<float4*>(&r_s[t][c]) = r4;
                    *reinterpret_cast<float4*>(&k_s[t][c]) = k4;
                    const float4 b = bw[n], e = ba[n];
                    *reinterpret_cast<float4*>(&w_s[t][c]) = ready ? zw :
                        make_float4(decay(zw.x + b.x), decay(zw.y + b.y), decay(zw.z + b.z), decay(zw.w + b.w));
                    *reinterpret_cast<float4*>(&a_s[t][c]) = ready ? za :
                        make_float4(sigmoid(za.x + e.x), sigmoid(za.y + e.y), sigmoid(za.z + e.z), sigmoid(za.w + e.w));
                    sk[i] = fmaf(k4.x, k4.x, sk[i]); sk[i] = fmaf(k4.y, k4.y, sk[i]);
                    sk[i] = fmaf(k4.z, k4.z, sk[i]); sk[i] = fmaf(k4.w, k4.w, sk[i]);
                }
                raw_arrived(pv[i]);
                v_s[t][lane] = raw1_f32<T>(pv[i]);
            } else if (t < tc) {
                const size_t at = (size_t)(start + t0 + t);
                const T* row = rkv + at * ld;
                for (int c = lane; c < DP; c += 32) {
                    const bool in = c < d;
                    const float kv = in ? to_f32(row[k_off + h * d + c]) : 0.f;
                    r_s[t][c] = in ? to_f32(row[r_off + h * d + c]) : 0.f;
                    k_s[t][c] = kv;
                    const float zw = in ? wl[at * ldw + h * d + c] : 0.f, za = in ? al[at * lda + h * d + c] : 0.f;
                    w_s[t][c] = !in || ready ? zw : decay(zw + w0[h * d + c]);
                    a_s[t][c] = !in || ready ? za : sigmoid(za + a0[h * d + c]);
                    sk[i] = fmaf(kv, kv, sk[i]);
                }
                v_s[t][lane] = v0 + lane < dv ? to_f32(row[v_off + h * dv + v0 + lane]) : 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < TPW; ++i) sk[i] = warp_sum(sk[i]);
        float mine = sk[0];                                // a lane per token divides
#pragma unroll
        for (int i = 1; i < TPW; ++i) mine = lane == i ? sk[i] : mine;
        if (lane < TPW) inv_s[warp + WARPS * lane] = 1.f / (mine + unit_eps);
        __syncthreads();
        if (vec && t0 + TC < len) fetch(t0 + TC);
        // y of the chunk's first token; every later one is summed while the token before it is written
        f32x2 kk[R / 2];
        f32x2 ya0 = 0ull, ya1 = 0ull, yb0 = 0ull, yb1 = 0ull;      // four chains to a column instead of one of R dependent steps
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(&k_s[0][KEY_OF(i, part)]);
            kk[2 * i] = k2.x; kk[2 * i + 1] = k2.y;
            ya0 = fma2(Sa[2 * i], k2.x, ya0); ya1 = fma2(Sa[2 * i + 1], k2.y, ya1);
            yb0 = fma2(Sb[2 * i], k2.x, yb0); yb1 = fma2(Sb[2 * i + 1], k2.y, yb1);
        }
        auto token = [&](int t, float& oa, float& ob) {
            const float inv = inv_s[t];
            const float za = part_sum<P>(sum2(ya0, ya1)) * inv, zb = part_sum<P>(sum2(yb0, yb1)) * inv;
            const f32x2 nza = both2(-za), nzb = both2(-zb), va = both2(v_s[t][vl]), vb = both2(v_s[t][vl + SCAN_HALF]);
            const int tn = t + 1 < tc ? t + 1 : t;         // the chunk's last token sums against nothing that is used
            f32x2 oa0 = 0ull, oa1 = 0ull, ob0 = 0ull, ob1 = 0ull;
            ya0 = ya1 = yb0 = yb1 = 0ull;
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 ww = *reinterpret_cast<const ulonglong2*>(&w_s[t][KEY_OF(i, part)]);
                const ulonglong2 aa = *reinterpret_cast<const ulonglong2*>(&a_s[t][KEY_OF(i, part)]);
                const ulonglong2 rr = *reinterpret_cast<const ulonglong2*>(&r_s[t][KEY_OF(i, part)]);
                const ulonglong2 kn = *reinterpret_cast<const ulonglong2*>(&k_s[tn][KEY_OF(i, part)]);
                Sa[2 * i] = fma2(ww.x, Sa[2 * i], mul2(kk[2 * i], fma2(aa.x, nza, va)));
                Sa[2 * i + 1] = fma2(ww.y, Sa[2 * i + 1], mul2(kk[2 * i + 1], fma2(aa.y, nza, va)));
                Sb[2 * i] = fma2(ww.x, Sb[2 * i], mul2(kk[2 * i], fma2(aa.x, nzb, vb)));
                Sb[2 * i + 1] = fma2(ww.y, Sb[2 * i + 1], mul2(kk[2 * i + 1], fma2(aa.y, nzb, vb)));
                ya0 = fma2(Sa[2 * i], kn.x, ya0); ya1 = fma2(Sa[2 * i + 1], kn.y, ya1);
                yb0 = fma2(Sb[2 * i], kn.x, yb0); yb1 = fma2(Sb[2 * i + 1], kn.y, yb1);
                oa0 = fma2(Sa[2 * i], rr.x, oa0); oa1 = fma2(Sa[2 * i + 1], rr.y, oa1);
                ob0 = fma2(Sb[2 * i], rr.x, ob0); ob1 = fma2(Sb[2 * i + 1], rr.y, ob1);
                kk[2 * i] = kn.x; kk[2 * i + 1] = kn.y;
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
        __syncthreads();
        float* o_row = out + (size_t)(start + t0 + warp) * H * dv + h * dv + v0 + lane;
#pragma unroll
        for (int i = 0; i < TPW; ++i)
            if (warp + WARPS * i < tc && v0 + lane < dv) o_row[(size_t)i * WARPS * H * dv] = o_s[warp + WARPS * i][lane];
    }
    if (live_a) scan_store_pairs<R, P>(Sa, st + (size_t)vl * DP, part);
    if (live_b) scan_store_pairs<R, P>(Sb, st + (size_t)(vl + SCAN_HALF) * DP, part);
}

// rkv: T [n, ld], r of head h at column r_off + h d, k at k_off + h d, v at v_off + h dv.  wl, al: float32 logits of the
// decay and of the removal rate, [n, ldw] and [n, lda] with H d columns; w0, a0 float32 [H d] (`ready`: the decays and
// rates themselves, the biases are not read).  out float32 [n, H dv].
extern "C" int gi_general_delta_scan(const void* rkv, long long ld, int act_dtype, int r_off, int k_off, int v_off,
                                     const float* wl, long long ldw, const float* w0, const float* al, long long lda,
                                     const float* a0, float unit_eps, float* state, long long state_stride,
                                     const int* spans, const int* tok_slot, float* out, int n_seq, int H, int d, int dv,
                                     int ready, void* stream) {
    const int DP = scan_padded(d);
    GI_REQUIRE(n_seq >= 0 && H > 0 && d > 0 && dv > 0 && DP > 0, "gi_general_delta_scan: key dimension %d (at most 256)", d);
    GI_REQUIRE(H <= 65535 && (dv + SCAN_VS - 1) / SCAN_VS <= 65535, "gi_general_delta_scan: %d heads of %d values", H, dv);
    GI_REQUIRE(ldw >= (long long)H * d && lda >= (long long)H * d, "gi_general_delta_scan: logits narrower than %d heads of %d", H, d);
    GI_REQUIRE(state_stride >= (long long)H * dv * DP && state_stride % 4 == 0, "gi_general_delta_scan: state rows of %lld "
               "floats are shorter than %lld or no multiple of 4", state_stride, (long long)H * dv * DP);
    if (n_seq == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(n_seq, H, (dv + SCAN_VS - 1) / SCAN_VS);
    const int esz = act_dtype == GI_DTYPE_F32 ? 4 : 2;
    auto on16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    const int vec = d % 4 == 0 && ld % 4 == 0 && r_off % 4 == 0 && k_off % 4 == 0 && ldw % 4 == 0 && lda % 4 == 0 &&
                    (uintptr_t)rkv % (4 * esz) == 0 && on16(wl) && on16(al) && on16(w0) && on16(a0);
#define GD_LAUNCH(T, R, P)                                                                                            \
    gi_launch(general_delta_scan_kernel<T, R, P>, grid, dim3(SCAN_HALF * P), 0, s, (const T*)rkv, ld, r_off, k_off, v_off, \
              wl, ldw, w0, al, lda, a0, unit_eps, state, state_stride, spans, tok_slot, out, H, d, dv, vec, ready)
    if (act_dtype == GI_DTYPE_F32) SCAN_SIZES(GD_LAUNCH, float)
    else if (act_dtype == GI_DTYPE_BF16) SCAN_SIZES(GD_LAUNCH, bf16)
    else GI_REQUIRE(false, "gi_general_delta_scan: activation dtype %d", act_dtype);
#undef GD_LAUNCH
    return gi_check_launch("gi_general_delta_scan");
}
