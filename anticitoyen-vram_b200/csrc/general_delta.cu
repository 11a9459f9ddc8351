// A linear recurrence with a generalized delta rule: a decay and a removal rate for every key channel.
//
// Per (request, head), S: [D, D] float in a state slot (rows: key channels, columns: value channels), u = k / sqrt(sum(k^2) + 1e-6):
//
//     S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,        o_t = S_t^T r_t
//
// A token's row of the input product is [r | k | v | z | g | x] (I = H*D each, then L): z the removal rate in front of its
// sigmoid, g the output gate in front of its sigmoid, x the decay's inner values in front of their tanh.  All float.
//
//   acv_delta_prepare   w[t][c] = exp(-exp(-1/2) sigmoid(w0[c] + sum_j W2[c][j] tanh(x[t][j])));  z becomes
//                       al = sigmoid(z) u in place;  per (token, head): 1 / sqrt(sum(k^2) + 1e-6), and <k_{t+1}, al_t>
//   acv_delta           the recurrence for portions and single tokens, o float
//   acv_delta_step      steps in which every request brings one token: all of the above, the head's norm, weight and gate
//                       in one launch
//
// acv_delta.  A column of S is a recurrence of its own, S[:, c].  G lanes of a warp share a column (R rows each, in
// registers); a block of four warps holds 4 * 32 / G columns and walks the tokens in chunks staged in shared memory, the next
// chunk copied while one is computed.  What bounds a token's time is the chain product with u -> sum over the lanes
// -> update -> next product; it is cut in half by looking one token ahead.  With X_t = diag(w_t) S_{t-1} + k_t v_t^T (known
// before p_t = u_t^T S_{t-1} is):
//
//     S_t = X_t - al_t p_t,     p_{t+1} = n_{t+1} (k_{t+1}^T X_t - <k_{t+1}, al_t> p_t)       n = 1 / sqrt(sum(k^2) + 1e-6)
//
// so the lanes' sum of k_{t+1}^T X_t runs beside token t's own update; <k_{t+1}, al_t> is a number per token and head.
#include "mma_tiles.cuh"

#define DL_WARPS 4
#define DL_RATE 0.6065306597126334f         // exp(-1/2)
#define DL_UNIT_EPS 1e-6f

__device__ __forceinline__ float dl_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// ----------------------------------------------------------------------------- decays, removal vectors
#define DP_TOK 8
// grid (tiles of DP_TOK tokens, tiles of whole heads).  proj: rows of `ld` floats; w2t float [L][I].  Half of the block's
// threads take the first four tokens' decays, half the others; then a warp a (token, head).
__global__ void __launch_bounds__(256)
delta_prepare_kernel(float* __restrict__ proj, int ld, const float* __restrict__ w2t, const float* __restrict__ w0,
                     float* __restrict__ w, float2* __restrict__ sc, int T_tokens, int H, int D, int L, int heads_per) {
    extern __shared__ __align__(16) float th[];         // [L][DP_TOK]
    pdl_wait();
    const int I = H * D;
    const int t0 = blockIdx.x * DP_TOK;
    const int n = min(DP_TOK, T_tokens - t0);
    const int h0 = blockIdx.y * heads_per, h1 = min(H, h0 + heads_per);
    for (int i = threadIdx.x; i < L * DP_TOK; i += blockDim.x) {
        const int tt = i / L, j = i - tt * L;
        th[j * DP_TOK + tt] = tt < n ? tanhf(proj[(size_t)(t0 + tt) * ld + 5 * (size_t)I + j]) : 0.f;
    }
    __syncthreads();
    const int half = threadIdx.x >> 7;
    for (int c = h0 * D + (threadIdx.x & 127); c < h1 * D; c += 128) {
        const float z0 = w0[c];
        float z[4] = {z0, z0, z0, z0};
#pragma unroll 8
        for (int j = 0; j < L; ++j) {
            const float m = w2t[(size_t)j * I + c];
            const float4 x = *reinterpret_cast<const float4*>(th + j * DP_TOK + half * 4);
            z[0] = fmaf(m, x.x, z[0]); z[1] = fmaf(m, x.y, z[1]); z[2] = fmaf(m, x.z, z[2]); z[3] = fmaf(m, x.w, z[3]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (half * 4 + i < n) w[(size_t)(t0 + half * 4 + i) * I + c] = expf(-DL_RATE * dl_sigmoid(z[i]));
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    for (int u = warp; u < n * (h1 - h0); u += nw) {
        const int tt = u / (h1 - h0), h = h0 + u - tt * (h1 - h0), t = t0 + tt;
        const float* k = proj + (size_t)t * ld + I + (size_t)h * D;
        const float* kn = t + 1 < T_tokens ? k + ld : k;        // (behind the last token: never used)
        float* z = proj + (size_t)t * ld + 3 * (size_t)I + (size_t)h * D;
        // one pass: the removal vector without its inverse root, and both sums
        float ss = 0.f, dot = 0.f;
        for (int e = lane; e < D; e += 32) {
            const float kk = k[e], al = dl_sigmoid(z[e]) * kk;
            ss = fmaf(kk, kk, ss);
            dot = fmaf(kn[e], al, dot);
        }
        ss = warp_sum(ss);
        dot = warp_sum(dot);
        const float inv = 1.f / sqrtf(ss + DL_UNIT_EPS);
        for (int e = lane; e < D; e += 32) z[e] = dl_sigmoid(z[e]) * (k[e] * inv);
        if (lane == 0) sc[(size_t)t * H + h] = make_float2(inv, dot * inv);
    }
    // the recurrence has few, long-lived blocks: begun while these blocks fill the SMs they would pile up on whichever
    // SMs have room first
    pdl_launch_dependents();
}

// proj: float [T][ld], rows [r | k | v | z | g | x]; w: float [T][H*D]; sc: float2 [T][H].
ACV_API int acv_delta_prepare(float* proj, int ld, const float* w2t, const float* w0, float* w, float* sc, int T_tokens, int H,
                              int D, int L, cudaStream_t stream) {
    if (T_tokens <= 0) return 0;
    if (H <= 0 || D <= 0 || L <= 0 || L > 1024 || ld < 5 * H * D + L) return ACV_ERR_SIZE;
    int heads_per = 128 / D;
    heads_per = heads_per < 1 ? 1 : (heads_per > H ? H : heads_per);
    const dim3 grid((T_tokens + DP_TOK - 1) / DP_TOK, (H + heads_per - 1) / heads_per);
    if (grid.y > 65535) return ACV_ERR_SIZE;
    acv_launch(PDL_MISC, delta_prepare_kernel, grid, 256, (size_t)L * DP_TOK * sizeof(float), stream, proj, ld, w2t, w0, w,
               (float2*)sc, T_tokens, H, D, L, heads_per);
    return acv_launch_status();
}

// ----------------------------------------------------------------------------- the recurrence
// two floats that one instruction works on
typedef unsigned long long f2;
__device__ __forceinline__ f2 f2_pack(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float f2_total(f2 x) {
    float a, b;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(x));
    return a + b;
}
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

template <int G>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = 1; o < G; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// The sums over the G lanes of a column of eight values each: every step halves the values that a lane still carries,
// so eight sums cost 7 exchanges at G = 8.  Afterwards v[0 .. 8/min(G,8)) of a lane are the totals of the values
// eight_first(lane) + i.
template <int G>
__device__ __forceinline__ void lanes_sum8(float (&v)[8], int lane) {
    if constexpr (G > 1) {
        const bool up = lane & 1;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float keep = up ? v[i + 4] : v[i], give = up ? v[i] : v[i + 4];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
        }
    }
    if constexpr (G > 2) {
        const bool up = lane & 2;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float keep = up ? v[i + 2] : v[i], give = up ? v[i] : v[i + 2];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
        }
    }
    if constexpr (G > 4) {
        const bool up = lane & 4;
        const float keep = up ? v[1] : v[0], give = up ? v[0] : v[1];
        v[0] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
    }
#pragma unroll
    for (int o = 8; o < G; o <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
}
template <int G>
__device__ __forceinline__ int eight_first(int lane) {
    return (G > 1 ? (lane & 1) * 4 : 0) + (G > 2 ? (lane & 2) : 0) + (G > 4 ? (lane & 4) >> 2 : 0);
}

// R rows and C neighbouring columns of S a thread, G lanes a column group, NW warps a block
template <int R, int G, int C, int NW>
__global__ void __launch_bounds__(NW * 32)
delta_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ w, const float2* __restrict__ sc,
             float* __restrict__ state, const int* __restrict__ slots, const int* __restrict__ cu_q, float* __restrict__ o,
             int H, int D, int TC, int vec) {
    constexpr int DP = R * G, DVT = NW * (32 / G) * C, R2 = R / 2;
    extern __shared__ __align__(16) float sm[];
    const int set = TC * (4 * DP + DVT + 2) + DP;       // floats of a staged chunk (k has one row more)
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * DVT;
    const int tid = threadIdx.x, nthr = NW * 32, lane = tid & 31, warp = tid >> 5;
    if (DP != D || c0 + DVT > D)                        // columns that no copy writes read as zeros
        for (int i = tid; i < 2 * set; i += nthr) sm[i] = 0.f;
    pdl_wait();
    const int t0 = cu_q[seq], t1 = cu_q[seq + 1];
    if (t1 <= t0) return;
    const int g = lane % G, cl = (warp * (32 / G) + lane / G) * C, c = c0 + cl;
    const int I = H * D;
    float* st = state + ((size_t)slots[seq] * H + h) * D * D;
    const float* base = proj + (size_t)h * D;

    auto stage = [&](int tb, float* s) {
        const int n = min(TC, t1 - tb);
        float* rs = s; float* ws_ = rs + TC * DP; float* as_ = ws_ + TC * DP; float* ks = as_ + TC * DP;
        float* vs = ks + (TC + 1) * DP; float* ss = vs + TC * DVT;
        if (vec) {
            const int d4 = D >> 2;
            for (int i = tid; i < (n + 1) * d4; i += nthr) {
                const int tt = i / d4, e = (i - tt * d4) << 2, t = tb + tt;
                const float* row = base + (size_t)t * ld + e;
                const bool in = t < t1;
                cp_async16(smem_u32(ks + tt * DP + e), in ? (const void*)(row + I) : (const void*)proj, in);
                if (tt < n) {
                    cp_async16(smem_u32(rs + tt * DP + e), row, true);
                    cp_async16(smem_u32(as_ + tt * DP + e), row + 3 * (size_t)I, true);
                    cp_async16(smem_u32(ws_ + tt * DP + e), w + (size_t)t * I + (size_t)h * D + e, true);
                }
            }
            for (int i = tid; i < n * (DVT >> 2); i += nthr) {
                const int tt = i / (DVT >> 2), e = (i - tt * (DVT >> 2)) << 2;
                const bool in = c0 + e < D;
                cp_async16(smem_u32(vs + tt * DVT + e), in ? (const void*)(base + (size_t)(tb + tt) * ld + 2 * (size_t)I + c0 + e) : (const void*)proj, in);
            }
        } else {
            for (int i = tid; i < (n + 1) * D; i += nthr) {
                const int tt = i / D, e = i - tt * D, t = tb + tt;
                const float* row = base + (size_t)t * ld + e;
                ks[tt * DP + e] = t < t1 ? row[I] : 0.f;
                if (tt < n) {
                    rs[tt * DP + e] = row[0];
                    as_[tt * DP + e] = row[3 * (size_t)I];
                    ws_[tt * DP + e] = w[(size_t)t * I + (size_t)h * D + e];
                }
            }
            for (int i = tid; i < n * DVT; i += nthr) {
                const int tt = i / DVT, e = i - tt * DVT;
                vs[i] = c0 + e < D ? base[(size_t)(tb + tt) * ld + 2 * (size_t)I + c0 + e] : 0.f;
            }
        }
        for (int tt = tid; tt < n; tt += nthr) reinterpret_cast<float2*>(ss)[tt] = sc[(size_t)(tb + tt) * H + h];
    };

    // a thread's rows: pairs of neighbours, four neighbours to a 16-byte piece, pieces G apart
    f2 S[C][R2];
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < R2; ++i) {
            const int d = ((i >> 1) * G + g) * 4 + (i & 1) * 2;
            const bool in = c + j < D;
            S[j][i] = f2_pack(in && d < D ? st[(size_t)d * D + c + j] : 0.f, in && d + 1 < D ? st[(size_t)(d + 1) * D + c + j] : 0.f);
        }
    __syncthreads();            // (the zeros stand before the first copies)
    stage(t0, sm);
    cp_async_commit();
    auto rows = [&](const float* row, f2 (&x)[R2]) {
#pragma unroll
        for (int i = 0; i < R2; i += 2) {
            const ulonglong2 q = reinterpret_cast<const ulonglong2*>(row)[(i >> 1) * G + g];
            x[i] = q.x; x[i + 1] = q.y;
        }
    };
    auto dot = [&](const f2 (&x)[R2], const f2 (&y)[R2]) {
        f2 a = f2_mul(x[0], y[0]);
#pragma unroll
        for (int i = 1; i < R2; ++i) a = f2_fma(x[i], y[i], a);
        return f2_total(a);
    };
    f2 kc[R2];                  // the current token's key rows
    float q[C], p[C], cp = 0.f;
#pragma unroll
    for (int j = 0; j < C; ++j) q[j] = p[j] = 0.f;
    bool first = true;
    int turn = 0;
    for (int tb = t0; tb < t1; tb += TC, turn ^= 1) {
        const int n = min(TC, t1 - tb);
        float* s = sm + turn * set;
        // (the other set was read in the turn before this one, whose last barrier every thread has passed)
        if (tb + TC < t1) stage(tb + TC, sm + (turn ^ 1) * set);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* rs = s; const float* wsm = rs + TC * DP; const float* asm_ = wsm + TC * DP; const float* ks = asm_ + TC * DP;
        const float* vs = ks + (TC + 1) * DP + cl; const float2* ss = reinterpret_cast<const float2*>(ks + (TC + 1) * DP + TC * DVT);
        if (first) {
            first = false;
            rows(ks, kc);
#pragma unroll
            for (int j = 0; j < C; ++j) q[j] = lanes_sum<G>(dot(kc, S[j]));
        }
        // a token's own vectors, read one token ahead of their use
        struct Token { f2 w[R2], k[R2], al[R2], r[R2]; float v[C]; float2 nc; };
        auto fetch = [&](Token& x, int tt) {
            rows(wsm + tt * DP, x.w);
            rows(ks + (tt + 1) * DP, x.k);          // the key of the token behind it
            rows(asm_ + tt * DP, x.al);
            rows(rs + tt * DP, x.r);
#pragma unroll
            for (int j = 0; j < C; ++j) x.v[j] = vs[tt * DVT + j];
            x.nc = ss[tt];
        };
        // one token: from S_{t-1} and q = k_t^T X_{t-1} to S_t, this lane's part of o_t, and the next q, whose exchanges
        // between the lanes are issued among the work that does not wait for them
        auto token = [&](const Token& x, float (&part)[C]) {
            f2 X[C][R2];
            float d[C];
#pragma unroll
            for (int j = 0; j < C; ++j) {
                const f2 vv = f2_pack(x.v[j], x.v[j]);
#pragma unroll
                for (int i = 0; i < R2; ++i) X[j][i] = f2_fma(x.w[i], S[j][i], f2_mul(kc[i], vv));
            }
#pragma unroll
            for (int j = 0; j < C; ++j) d[j] = dot(x.k, X[j]);
            if constexpr (G > 1)
#pragma unroll
                for (int j = 0; j < C; ++j) d[j] += __shfl_xor_sync(0xffffffffu, d[j], 1);
#pragma unroll
            for (int j = 0; j < C; ++j) {
                p[j] = x.nc.x * fmaf(-cp, p[j], q[j]);
                const f2 np = f2_pack(-p[j], -p[j]);
#pragma unroll
                for (int i = 0; i < R2; ++i) S[j][i] = f2_fma(x.al[i], np, X[j][i]);
            }
            if constexpr (G > 2)
#pragma unroll
                for (int j = 0; j < C; ++j) d[j] += __shfl_xor_sync(0xffffffffu, d[j], 2);
#pragma unroll
            for (int j = 0; j < C; ++j) part[j] = dot(x.r, S[j]);
#pragma unroll
            for (int o = 4; o < G; o <<= 1)
#pragma unroll
                for (int j = 0; j < C; ++j) d[j] += __shfl_xor_sync(0xffffffffu, d[j], o);
#pragma unroll
            for (int j = 0; j < C; ++j) q[j] = d[j];
#pragma unroll
            for (int i = 0; i < R2; ++i) kc[i] = x.k[i];
            cp = x.nc.y;
        };
        int tt = 0;
        Token a;
        fetch(a, 0);
        for (; tt + 8 <= n; tt += 8) {
            float part[C][8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                Token b;
                fetch(b, min(tt + i + 1, TC - 1));
                float one[C];
                token(a, one);
                a = b;
#pragma unroll
                for (int j = 0; j < C; ++j) part[j][i] = one[j];
            }
            constexpr int LEFT = G >= 8 ? 1 : 8 / G;
#pragma unroll
            for (int j = 0; j < C; ++j) {
                lanes_sum8<G>(part[j], lane);
                if ((G <= 8 || g < 8) && c + j < D) {
                    float* dst = o + (size_t)(tb + tt + eight_first<G>(lane)) * I + (size_t)h * D + c + j;
#pragma unroll
                    for (int i = 0; i < LEFT; ++i) dst[(size_t)i * I] = part[j][i];
                }
            }
        }
        for (; tt < n; ++tt) {
            float one[C];
            fetch(a, tt);
            token(a, one);
#pragma unroll
            for (int j = 0; j < C; ++j) {
                one[j] = lanes_sum<G>(one[j]);
                if (g == 0 && c + j < D) o[(size_t)(tb + tt) * I + (size_t)h * D + c + j] = one[j];
            }
        }
        __syncthreads();
    }
    pdl_launch_dependents();
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < R2; ++i) {
            const int d = ((i >> 1) * G + g) * 4 + (i & 1) * 2;
            float a, b;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(S[j][i]));
            if (c + j < D && d < D) st[(size_t)d * D + c + j] = a;
            if (c + j < D && d + 1 < D) st[(size_t)(d + 1) * D + c + j] = b;
        }
}

template <int R, int G, int C, int NW>
static int launch_delta(const float* proj, int ld, const float* w, const float2* sc, float* state, const int* slots,
                        const int* cu_q, float* o, int n_seqs, int H, int D, cudaStream_t stream) {
    constexpr int DP = R * G, DVT = NW * (32 / G) * C;
    const int per_token = (4 * DP + DVT + 2) * 4;
    int TC = 32;
    while (TC > 8 && 2 * (TC * per_token + DP * 4) > 72 * 1024) TC -= 8;
    const size_t smem = 2 * ((size_t)TC * per_token + DP * 4);
    static AcvSmemConfig cfg;
    if (smem > 48 * 1024)
        if (int e = acv_ensure_smem(cfg, delta_kernel<R, G, C, NW>, (int)smem)) return e;
    const int vec = D % 4 == 0 && ld % 4 == 0 && !((uintptr_t)proj & 15) && !((uintptr_t)w & 15);
    const dim3 grid(n_seqs, H, (D + DVT - 1) / DVT);
    if (grid.y > 65535 || grid.z > 65535) return ACV_ERR_SIZE;
    acv_launch(PDL_ATTN, delta_kernel<R, G, C, NW>, grid, NW * 32, smem, stream, proj, ld, w, sc, state, slots, cu_q, o, H, D, TC, vec);
    return acv_launch_status();
}

// After acv_delta_prepare.  o: float [T][H*D]; state: float [slots][H][D][D]; heads of up to 512 channels.
// form: 0 by the sizes; 1, 2, 3 (heads of 33 to 64 channels): one, two or four columns a thread.
ACV_API int acv_delta(const float* proj, int ld, const float* w, const float* sc, float* state, const int* slots,
                      const int* cu_q, float* o, int n_seqs, int H, int D, int form, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || D <= 0 || D > 512) return ACV_ERR_SIZE;
#define DL_CASE(RR, GG, CC, WW) \
    return launch_delta<RR, GG, CC, WW>(proj, ld, w, (const float2*)sc, state, slots, cu_q, o, n_seqs, H, D, stream);
    if (D <= 8) DL_CASE(8, 1, 1, 4)
    if (D <= 16) DL_CASE(8, 2, 1, 4)
    if (D <= 32) DL_CASE(8, 4, 1, 4)
    if (D <= 64) {
        if (form == 1) DL_CASE(8, 8, 1, 4)
        if (form == 3) DL_CASE(8, 8, 4, 2)
        if (form == 4) DL_CASE(4, 16, 2, 4)
        if (form == 5) DL_CASE(8, 8, 2, 4)
        if (form == 6) DL_CASE(4, 16, 4, 2)
        if (form == 7) DL_CASE(8, 8, 4, 1)
        if (form == 8) DL_CASE(16, 4, 1, 2)
        DL_CASE(8, 8, 2, 2)
    }
    if (D <= 128) {
        if (form == 1) DL_CASE(8, 16, 1, 4)
        if (form == 2) DL_CASE(8, 16, 4, 2)
        if (form == 3) DL_CASE(16, 8, 2, 2)
        DL_CASE(8, 16, 2, 4)
    }
    if (D <= 256) DL_CASE(8, 32, 1, 4)
    DL_CASE(16, 32, 1, 4)
#undef DL_CASE
}

// ----------------------------------------------------------------------------- one token a request, everything
// A block of 256 threads a (request, head).  A thread holds RPT rows of four neighbouring columns: c4 = D / 4 threads cover a
// row, NG = 256 / c4 groups of rows stand side by side; sums over rows pass through shared memory.
template <typename T, int RPT>
__global__ void __launch_bounds__(256)
delta_step_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ w2t, const float* __restrict__ w0,
                  const float* __restrict__ weight, float eps, float* __restrict__ state, const int* __restrict__ slots,
                  const int* __restrict__ cu_q, T* __restrict__ out, int ldo, int H, int D, int L) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    float* rs = sm; float* ks = rs + D; float* vs = ks + D; float* as_ = vs + D; float* ws = as_ + D; float* ps = ws + D;
    float* part = ps + D;                   // [max(NG, 256 / D + 1)][D]
    const int c4n = D >> 2, NG = 256 / c4n;
    float* th = part + (size_t)(NG > 256 / D + 1 ? NG : 256 / D + 1) * D;      // [L]
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int t = cu_q[seq], I = H * D;
    float* st = state + ((size_t)slots[seq] * H + h) * D * D;
    const int g = tid / c4n, col = (tid - g * c4n) << 2;
    const bool owner = g < NG;
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + i * NG;
        S[i] = owner && d < D ? *reinterpret_cast<const float4*>(st + (size_t)d * D + col) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float* row = proj + (size_t)t * ld + (size_t)h * D;
    for (int e = tid; e < D; e += 256) {
        rs[e] = row[e];
        ks[e] = row[(size_t)I + e];
        vs[e] = row[2 * (size_t)I + e];
        as_[e] = row[3 * (size_t)I + e];
    }
    for (int j = tid; j < L; j += 256) th[j] = tanhf(proj[(size_t)t * ld + 5 * (size_t)I + j]);
    __syncthreads();
    // the decays: 256 / D threads share a channel's sum
    const int np = 256 / D;                 // (D <= 128)
    const int pp = tid / D, pc = tid - pp * D;
    if (pp < np) {
        float z = 0.f;
        const float* m = w2t + (size_t)h * D + pc;
        for (int j = pp; j < L; j += np) z = fmaf(m[(size_t)j * I], th[j], z);
        part[(size_t)pp * D + pc] = z;
    }
    float ss = 0.f;
    for (int e = lane; e < D; e += 32) ss = fmaf(ks[e], ks[e], ss);
    const float inv = 1.f / sqrtf(warp_sum(ss) + DL_UNIT_EPS);         // (every warp for itself)
    __syncthreads();
    if (tid < D) {
        float z = w0[(size_t)h * D + tid];
        for (int i = 0; i < np; ++i) z += part[(size_t)i * D + tid];
        ws[tid] = expf(-DL_RATE * dl_sigmoid(z));
        as_[tid] = dl_sigmoid(as_[tid]) * (ks[tid] * inv);
    }
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + i * NG;
        if (owner && d < D) {
            const float k = ks[d];
            acc.x = fmaf(k, S[i].x, acc.x); acc.y = fmaf(k, S[i].y, acc.y);
            acc.z = fmaf(k, S[i].z, acc.z); acc.w = fmaf(k, S[i].w, acc.w);
        }
    }
    if (owner) *reinterpret_cast<float4*>(part + (size_t)g * D + col) = acc;
    __syncthreads();
    if (tid < D) {
        float p = 0.f;
        for (int i = 0; i < NG; ++i) p += part[(size_t)i * D + tid];
        ps[tid] = p * inv;
    }
    __syncthreads();
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner) {
        const float4 p = *reinterpret_cast<const float4*>(ps + col), v = *reinterpret_cast<const float4*>(vs + col);
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int d = g + i * NG;
            if (d < D) {
                const float wd = ws[d], ad = as_[d], kd = ks[d], rd = rs[d];
                S[i].x = fmaf(-ad, p.x, fmaf(wd, S[i].x, kd * v.x)); S[i].y = fmaf(-ad, p.y, fmaf(wd, S[i].y, kd * v.y));
                S[i].z = fmaf(-ad, p.z, fmaf(wd, S[i].z, kd * v.z)); S[i].w = fmaf(-ad, p.w, fmaf(wd, S[i].w, kd * v.w));
                *reinterpret_cast<float4*>(st + (size_t)d * D + col) = S[i];
                acc.x = fmaf(rd, S[i].x, acc.x); acc.y = fmaf(rd, S[i].y, acc.y);
                acc.z = fmaf(rd, S[i].z, acc.z); acc.w = fmaf(rd, S[i].w, acc.w);
            }
        }
        *reinterpret_cast<float4*>(part + (size_t)g * D + col) = acc;
    }
    __syncthreads();
    float ov = 0.f;
    if (tid < D)
        for (int i = 0; i < NG; ++i) ov += part[(size_t)i * D + tid];
    const float inv_rms = 1.f / sqrtf(block_sum(ov * ov, red) / (float)D + eps);
    if (tid < D) {
        const float gate = row[4 * (size_t)I + tid];
        out[(size_t)t * ldo + (size_t)h * D + tid] = from_f32<T>(ov * inv_rms * weight[(size_t)h * D + tid] * dl_sigmoid(gate));
    }
}

static size_t delta_step_smem(int D, int L) {
    const int NG = 256 / (D / 4), np = 256 / D + 1;
    return (size_t)(6 * D + (NG > np ? NG : np) * D + L) * sizeof(float);
}

// 1 if acv_delta_step runs these sizes
ACV_API int acv_delta_step_takes(int D, int L) { return D >= 4 && D % 4 == 0 && D <= 128 && L > 0 && delta_step_smem(D, L) <= 48 * 1024; }

// out: rows of H*D elements at ldo (float or bfloat16): each head's o / sqrt(mean(o^2) + eps), times weight (float [H*D]),
// times sigmoid(g).  proj as acv_delta_prepare takes it (not prepared); every request brings one token.
ACV_API int acv_delta_step(const float* proj, int ld, const float* w2t, const float* w0, const float* weight, float eps,
                           float* state, const int* slots, const int* cu_q, void* out, int ldo, int n_seqs, int H, int D,
                           int L, int dtype, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || H > 65535 || !acv_delta_step_takes(D, L) || ld < 5 * H * D + L) return ACV_ERR_SIZE;
    if ((uintptr_t)state & 15) return ACV_ERR_ALIGN;
    const int NG = 256 / (D / 4), rows = (D + NG - 1) / NG;
    const size_t smem = delta_step_smem(D, L);
    const dim3 grid(n_seqs, H);
#define DS_CASE(N)                                                                                                          \
    if (rows <= N) {                                                                                                        \
        if (dtype == ACV_F32)                                                                                               \
            acv_launch(PDL_ATTN, delta_step_kernel<float, N>, grid, 256, smem, stream, proj, ld, w2t, w0, weight, eps, state, \
                       slots, cu_q, (float*)out, ldo, H, D, L);                                                             \
        else if (dtype == ACV_BF16)                                                                                         \
            acv_launch(PDL_ATTN, delta_step_kernel<bf16, N>, grid, 256, smem, stream, proj, ld, w2t, w0, weight, eps, state,  \
                       slots, cu_q, (bf16*)out, ldo, H, D, L);                                                              \
        else                                                                                                                \
            return ACV_ERR_DTYPE;                                                                                           \
        return acv_launch_status();                                                                                         \
    }
    DS_CASE(1) DS_CASE(2) DS_CASE(4) DS_CASE(8) DS_CASE(16)
#undef DS_CASE
    return ACV_ERR_SIZE;
}
