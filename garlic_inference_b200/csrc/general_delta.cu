// The generalized delta rule: a decay and a removal rate per head and key channel, float32 state per head.
//
//   w = exp(-exp(-1/2) sigmoid(zw + w0)),   a = sigmoid(za + a0),   u = k / sqrt(|k|^2 + eps)
//   S_t = diag(w) S_(t-1) - (a u)(u^T S_(t-1)) + k v^T        both terms on the old state
//   o_t = S_t^T r
//
// A block owns one (sequence, head, slice of 32 value columns) and walks the sequence's tokens of the step in order,
// like the other scans (recurrent.cu says what a thread holds).  With y = k^T S_(t-1) of a column and
// z = y / (|k|^2 + eps), channel c of the column becomes w_c S_c + k_c (v - a_c z).  The one sum over the keys that the
// next token waits for is y, so it is started while the present token is written: the loop that renews S also sums
// S against the next token's k.  The read-outs of P tokens are summed over the lanes together.
// NikolayBlagoev/garlic-inference has no recurrent mixer.
#include "scan.cuh"

#define GD_DECAY 0.60653065971263342f        // exp(-1/2)
#define GD_TC(DP) ((DP) <= 64 ? 32 : ((DP) <= 128 ? 16 : 8))       // tokens in shared memory at a time

template <typename T, int R, int P>
__global__ void __launch_bounds__(SCAN_VS * P)
general_delta_scan_kernel(const T* __restrict__ rkv, long long ld, int r_off, int k_off, int v_off,
                          const float* __restrict__ wl, long long ldw, const float* __restrict__ w0,
                          const float* __restrict__ al, long long lda, const float* __restrict__ a0, float unit_eps,
                          float* __restrict__ state, long long state_stride, const int* __restrict__ spans,
                          const int* __restrict__ tok_slot, float* __restrict__ out, int H, int d, int dv, int vec) {
    gi_pdl_start();
    constexpr int DP = R * P;
    constexpr int TC = GD_TC(DP);
    constexpr int THREADS = SCAN_VS * P, WARPS = P;
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
    const int part = threadIdx.x % P, vl = threadIdx.x / P, v = v0 + vl;
    const bool live = v < dv;
    if (slot < 0) {
        for (int t = 0; t < len; ++t)
            if (live && part == 0) out[(size_t)(start + t) * H * dv + h * dv + v] = 0.f;
        return;
    }
    float* st = state + (size_t)slot * state_stride + ((size_t)h * dv + (live ? v : 0)) * DP;
    float S[R];
    if (live) scan_load_state<R, P>(S, st, part);
    else {
#pragma unroll
        for (int e = 0; e < R; ++e) S[e] = 0.f;
    }
    typedef typename Raw4<T>::type raw_t;
    constexpr int TPW = TC / WARPS;
    constexpr int NQ = (DP / 4 + 31) / 32;
    raw_t pr[TPW][NQ], pk[TPW][NQ];
    float4 pw[TPW][NQ], pa[TPW][NQ];
    float pv[TPW];
    auto fetch = [&](int t0) {
        const int tc = min(TC, len - t0);
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = warp + WARPS * i;
            if (t >= tc) continue;
            const size_t at = (size_t)(start + t0 + t);
            const T* row = rkv + at * ld;
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                const int c = (lane + 32 * n) * 4;
                raw4_zero(pr[i][n]); raw4_zero(pk[i][n]); raw4_zero(pw[i][n]); raw4_zero(pa[i][n]);
                if (c < d) {
                    pr[i][n] = *reinterpret_cast<const raw_t*>(row + r_off + h * d + c);
                    pk[i][n] = *reinterpret_cast<const raw_t*>(row + k_off + h * d + c);
                    pw[i][n] = *reinterpret_cast<const float4*>(wl + at * ldw + h * d + c);
                    pa[i][n] = *reinterpret_cast<const float4*>(al + at * lda + h * d + c);
                }
            }
            pv[i] = v0 + lane < dv ? to_f32(row[v_off + h * dv + v0 + lane]) : 0.f;
        }
    };
    auto decay = [](float z) { return expf(-GD_DECAY * rc_sigmoid(z)); };
    if (vec) fetch(0);
    for (int t0 = 0; t0 < len; t0 += TC) {
        const int tc = min(TC, len - t0);
        __syncthreads();                                   // the last chunk's outputs and inputs are done with
        float sk[TPW];
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = warp + WARPS * i;
            sk[i] = 0.f;
            if (t >= tc) continue;
            if (vec) {
#pragma unroll
                for (int n = 0; n < NQ; ++n) {
                    const int c = (lane + 32 * n) * 4;
                    if (c >= DP) continue;
                    const float4 k4 = raw4_f32(pk[i][n]), zw = pw[i][n], za = pa[i][n];
                    *reinterpret_cast<float4*>(&r_s[t][c]) = raw4_f32(pr[i][n]);
                    *reinterpret_cast<float4*>(&k_s[t][c]) = k4;
                    float4 b = make_float4(0.f, 0.f, 0.f, 0.f), e = b;
                    if (c < d) { b = *reinterpret_cast<const float4*>(w0 + h * d + c); e = *reinterpret_cast<const float4*>(a0 + h * d + c); }
                    *reinterpret_cast<float4*>(&w_s[t][c]) = make_float4(decay(zw.x + b.x), decay(zw.y + b.y), decay(zw.z + b.z), decay(zw.w + b.w));
                    *reinterpret_cast<float4*>(&a_s[t][c]) = make_float4(rc_sigmoid(za.x + e.x), rc_sigmoid(za.y + e.y), rc_sigmoid(za.z + e.z), rc_sigmoid(za.w + e.w));
                    sk[i] = fmaf(k4.x, k4.x, sk[i]); sk[i] = fmaf(k4.y, k4.y, sk[i]);
                    sk[i] = fmaf(k4.z, k4.z, sk[i]); sk[i] = fmaf(k4.w, k4.w, sk[i]);
                }
                v_s[t][lane] = pv[i];
            } else {
                const size_t at = (size_t)(start + t0 + t);
                const T* row = rkv + at * ld;
                for (int c = lane; c < DP; c += 32) {
                    const bool in = c < d;
                    const float kv = in ? to_f32(row[k_off + h * d + c]) : 0.f;
                    r_s[t][c] = in ? to_f32(row[r_off + h * d + c]) : 0.f;
                    k_s[t][c] = kv;
                    w_s[t][c] = in ? decay(wl[at * ldw + h * d + c] + w0[h * d + c]) : 0.f;
                    a_s[t][c] = in ? rc_sigmoid(al[at * lda + h * d + c] + a0[h * d + c]) : 0.f;
                    sk[i] = fmaf(kv, kv, sk[i]);
                }
                v_s[t][lane] = v0 + lane < dv ? to_f32(row[v_off + h * dv + v0 + lane]) : 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = warp + WARPS * i;
            if (t >= tc) continue;
            const float sum = warp_sum(sk[i]);
            if (lane == 0) inv_s[t] = 1.f / (sum + unit_eps);
        }
        __syncthreads();
        if (vec && t0 + TC < len) fetch(t0 + TC);
        // y of the chunk's first token; every later one is summed while the token before it is written
        float4 kk[R / 4];
        float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            kk[i] = *reinterpret_cast<const float4*>(&k_s[0][KEY_OF(i, part)]);
            y0 = fmaf(S[4 * i], kk[i].x, y0); y1 = fmaf(S[4 * i + 1], kk[i].y, y1);
            y2 = fmaf(S[4 * i + 2], kk[i].z, y2); y3 = fmaf(S[4 * i + 3], kk[i].w, y3);
        }
        auto token = [&](int t) {
            const float z = part_sum<P>((y0 + y1) + (y2 + y3)) * inv_s[t];
            const float vt = v_s[t][vl];
            const int tn = t + 1 < tc ? t + 1 : t;         // the chunk's last token sums against nothing that is used
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
            y0 = y1 = y2 = y3 = 0.f;
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const float4 ww = *reinterpret_cast<const float4*>(&w_s[t][KEY_OF(i, part)]);
                const float4 aa = *reinterpret_cast<const float4*>(&a_s[t][KEY_OF(i, part)]);
                const float4 rr = *reinterpret_cast<const float4*>(&r_s[t][KEY_OF(i, part)]);
                const float4 kn = *reinterpret_cast<const float4*>(&k_s[tn][KEY_OF(i, part)]);
                S[4 * i] = fmaf(ww.x, S[4 * i], kk[i].x * fmaf(-aa.x, z, vt));
                S[4 * i + 1] = fmaf(ww.y, S[4 * i + 1], kk[i].y * fmaf(-aa.y, z, vt));
                S[4 * i + 2] = fmaf(ww.z, S[4 * i + 2], kk[i].z * fmaf(-aa.z, z, vt));
                S[4 * i + 3] = fmaf(ww.w, S[4 * i + 3], kk[i].w * fmaf(-aa.w, z, vt));
                y0 = fmaf(S[4 * i], kn.x, y0); y1 = fmaf(S[4 * i + 1], kn.y, y1);
                y2 = fmaf(S[4 * i + 2], kn.z, y2); y3 = fmaf(S[4 * i + 3], kn.w, y3);
                o0 = fmaf(S[4 * i], rr.x, o0); o1 = fmaf(S[4 * i + 1], rr.y, o1);
                o2 = fmaf(S[4 * i + 2], rr.z, o2); o3 = fmaf(S[4 * i + 3], rr.w, o3);
                kk[i] = kn;
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
        __syncthreads();
        for (int i = threadIdx.x; i < tc * SCAN_VS; i += THREADS) {
            const int tt = i / SCAN_VS, c = i - tt * SCAN_VS;
            if (v0 + c < dv) out[(size_t)(start + t0 + tt) * H * dv + h * dv + v0 + c] = o_s[tt][c];
        }
    }
    if (live) scan_store_state<R, P>(S, st, part);
}

// rkv: T [n, ld], r of head h at column r_off + h d, k at k_off + h d, v at v_off + h dv.  wl, al: float32 logits of the
// decay and of the removal rate, [n, ldw] and [n, lda] with H d columns; w0, a0 float32 [H d].  out float32 [n, H dv].
extern "C" int gi_general_delta_scan(const void* rkv, long long ld, int act_dtype, int r_off, int k_off, int v_off,
                                     const float* wl, long long ldw, const float* w0, const float* al, long long lda,
                                     const float* a0, float unit_eps, float* state, long long state_stride,
                                     const int* spans, const int* tok_slot, float* out, int n_seq, int H, int d, int dv,
                                     void* stream) {
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
    if (act_dtype == GI_DTYPE_F32) {
        SCAN_DISPATCH(general_delta_scan_kernel, float, (const float*)rkv, ld, r_off, k_off, v_off, wl, ldw, w0, al, lda, a0, unit_eps, state, state_stride, spans, tok_slot, out, H, d, dv, vec)
    } else if (act_dtype == GI_DTYPE_BF16) {
        SCAN_DISPATCH(general_delta_scan_kernel, bf16, (const bf16*)rkv, ld, r_off, k_off, v_off, wl, ldw, w0, al, lda, a0, unit_eps, state, state_stride, spans, tok_slot, out, H, d, dv, vec)
    } else {
        GI_REQUIRE(false, "gi_general_delta_scan: activation dtype %d", act_dtype);
    }
    return gi_check_launch("gi_general_delta_scan");
}
