// A linear recurrence with a generalized delta rule: a decay and a removal rate for every key channel.
//
// Per (request, head), S: [D, D] float in a state slot (rows: key channels, columns: value channels), u = k / sqrt(sum(k^2) + 1e-6):
//
//     S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,        o_t = S_t^T r_t
//
// A token's row of the input product is [r | k | v | z | g | x] (I = H*D each, then L): z the removal rate in front of its
// sigmoid, g the output gate in front of its sigmoid, x the decay's inner values in front of their tanh.  All float.
//
//   acv_delta_blocks    everything that does not need the state, for eight tokens of a request at a time
//   acv_delta           the recurrence over those blocks, o float (also over the blocks of csrc/gated_delta.cu, see there)
//   acv_delta_step      steps in which every request brings one token: all of the above, the head's norm, weight and gate
//                       in one launch
//
// Token by token the recurrence is a chain (product with u, a sum over the channels, an update, the next product) of some
// 300 cycles a token.  Eight tokens at once the state enters linearly.  With W_i the product of the block's decays up to
// token i (1..8, W_0 = 1; a decay is above 0.54, so W_8 is above 0.007 and may be divided by), al_i = a_i u_i, n_i the
// inverse root, S the state in front of the block, and over the block's tokens i, j
//
//     k'_i = n_i W_{i-1} k_i    r'_i = W_i r_i      kd_j = k_j / W_j      ad_j = al_j / W_j
//     K = low(k' kd^T)   A = low(k' ad^T)   (j < i)       P = low(r' kd^T)   Q = low(r' ad^T)   (j <= i)
//
// the products p_i = u_i^T S_{i-1} obey p = k' S + K v - A p, and o = r' S + P v - Q p.  Solved for the state (I + A is
// unit lower triangular; the solution is a forward substitution along the block's tokens, channel by channel):
//
//     kt = (I + A)^-1 k'    M = (I + A)^-1 K    rt = r' - Q kt    N = P - Q M
//     p = kt S + M v        o = rt S + N v      S_8 = W_8 (S + sum_j kd_j v_j^T - ad_j p_j^T)
//
// A block's record (floats, channels padded to DP with zeros): kt [8][DP], rt [8][DP], W_8 kd [8][DP], -W_8 ad [8][DP],
// W_8 [DP], M [8][8], N [8][8].  Tokens behind a portion's end are k = r = 0, w = 1: they change nothing.
#include "mma_tiles.cuh"

#define DL_TOK 8
#define DL_RATE 0.6065306597126334f         // exp(-1/2)
#define DL_UNIT_EPS 1e-6f

// (the quotient within two units in the last place; a denominator past 2^126 gives 0)
__device__ __forceinline__ float dl_sigmoid(float z) { return __fdividef(1.f, 1.f + expf(-z)); }

// channels of a head as a record pads them
static int delta_pad(int D) {
    int p = 8;
    while (p < D) p <<= 1;
    return p;
}
static size_t delta_record(int DP) { return (size_t)33 * DP + 128; }

// ----------------------------------------------------------------------------- the blocks' records
// grid (blocks of tokens, tiles of `heads` whole heads); a thread owns NC channels (tid + 256 q).  proj: rows of `ld` floats; w2t
// float [L][I]; rec: [items][H][record].
template <int NC>
__global__ void __launch_bounds__(256, NC == 1 ? 3 : 1)
delta_blocks_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ w2t, const float* __restrict__ w0,
                    const int* __restrict__ item_seq, const int* __restrict__ item_idx, const int* __restrict__ cu_q,
                    float* __restrict__ rec, int H, int D, int DP, int L, int heads) {
    extern __shared__ __align__(16) float sm[];
    const int PD = (D + 3) & ~3;            // pitch of a row of channels
    float* th = sm;                         // [L][8]
    float* mA = th + L * DL_TOK;            // [heads][16][PD]: raw k, then k', r'
    float* mB = mA + (size_t)heads * 16 * PD;       // [heads][16][PD]: kd, ad
    float* gm = mB + (size_t)heads * 16 * PD;       // [heads][16][16]: [K A; P Q]
    float* inv = gm + heads * 256;          // [heads][8]
    pdl_wait();
    const int item = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = item_seq[item], I = H * D;
    const int t0 = cu_q[seq] + item_idx[item] * DL_TOK;
    const int n = min(DL_TOK, cu_q[seq + 1] - t0);
    const int h0 = blockIdx.y * heads, nh = min(heads, H - h0);
    const float* base = proj + (size_t)t0 * ld;
    for (int i = tid; i < L * DL_TOK; i += 256) {
        const int tt = i / L, j = i - tt * L;
        th[j * DL_TOK + tt] = tt < n ? tanhf(base[(size_t)tt * ld + 5 * (size_t)I + j]) : 0.f;
    }
    float k[NC][DL_TOK], r[NC][DL_TOK], z[NC][DL_TOK], w[NC][DL_TOK];
#pragma unroll
    for (int q = 0; q < NC; ++q) {
        const int ch = tid + 256 * q, c = h0 * D + ch;
        const bool in = ch < nh * D;
#pragma unroll
        for (int tt = 0; tt < DL_TOK; ++tt) {
            const float* row = base + (size_t)tt * ld + c;
            const bool there = in && tt < n;
            r[q][tt] = there ? row[0] : 0.f;
            k[q][tt] = there ? row[I] : 0.f;
            z[q][tt] = there ? row[3 * (size_t)I] : 0.f;
        }
        if (in) {
            const int hh = ch / D, e = ch - hh * D;
#pragma unroll
            for (int tt = 0; tt < DL_TOK; ++tt) mA[((size_t)hh * 16 + tt) * PD + e] = k[q][tt];
        }
    }
    __syncthreads();
    for (int u = warp; u < nh * DL_TOK; u += 8) {
        const float* row = mA + ((size_t)(u >> 3) * 16 + (u & 7)) * PD;
        float ss = 0.f;
        for (int e = lane; e < D; e += 32) ss = fmaf(row[e], row[e], ss);
        ss = warp_sum(ss);
        if (lane == 0) inv[u] = 1.f / sqrtf(ss + DL_UNIT_EPS);
    }
#pragma unroll
    for (int q = 0; q < NC; ++q) {
        const int ch = tid + 256 * q, c = h0 * D + ch;
        const bool in = ch < nh * D;
        const float z0 = in ? w0[c] : 0.f;
#pragma unroll
        for (int tt = 0; tt < DL_TOK; ++tt) w[q][tt] = z0;
        if (in) {
#pragma unroll 8
            for (int j = 0; j < L; ++j) {
                const float m = w2t[(size_t)j * I + c];
                const float4 a = *reinterpret_cast<const float4*>(th + j * DL_TOK), b = *reinterpret_cast<const float4*>(th + j * DL_TOK + 4);
                w[q][0] = fmaf(m, a.x, w[q][0]); w[q][1] = fmaf(m, a.y, w[q][1]);
                w[q][2] = fmaf(m, a.z, w[q][2]); w[q][3] = fmaf(m, a.w, w[q][3]);
                w[q][4] = fmaf(m, b.x, w[q][4]); w[q][5] = fmaf(m, b.y, w[q][5]);
                w[q][6] = fmaf(m, b.z, w[q][6]); w[q][7] = fmaf(m, b.w, w[q][7]);
            }
        }
        float run = 1.f;                    // w becomes the running product W_i
#pragma unroll
        for (int tt = 0; tt < DL_TOK; ++tt) {
            if (tt < n) run *= expf(-DL_RATE * dl_sigmoid(w[q][tt]));
            w[q][tt] = run;
        }
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < NC; ++q) {
        const int ch = tid + 256 * q;
        if (ch < nh * D) {
            const int hh = ch / D, e = ch - hh * D;
            float* a = mA + (size_t)hh * 16 * PD + e;
            float* b = mB + (size_t)hh * 16 * PD + e;
#pragma unroll
            for (int tt = 0; tt < DL_TOK; ++tt) {
                const float over = __fdividef(1.f, w[q][tt]), ni = inv[hh * DL_TOK + tt];
                const float kp = ni * k[q][tt] * (tt ? w[q][tt - 1] : 1.f);
                r[q][tt] *= w[q][tt];
                z[q][tt] = dl_sigmoid(z[q][tt]) * (k[q][tt] * ni) * over;       // ad
                k[q][tt] *= over;                                               // kd
                a[tt * PD] = kp; a[(8 + tt) * PD] = r[q][tt];
                b[tt * PD] = k[q][tt]; b[(8 + tt) * PD] = z[q][tt];
            }
        }
    }
    if (PD != D)                            // the channels that fill a row's last 16 bytes
        for (int i = tid; i < nh * 32 * (PD - D); i += 256) {
            const int row = i / (PD - D), e = D + i % (PD - D);
            (row < nh * 16 ? mA + (size_t)row * PD : mB + (size_t)(row - nh * 16) * PD)[e] = 0.f;
        }
    __syncthreads();
    // [k'; r'] [kd; ad]^T, 16 x 16 for every head: a warp four of its rows, eight lanes share the channels of a 4 x 4 tile
    for (int u = warp; u < nh * 4; u += 8) {
        const int hh = u >> 2, ti = u & 3, tj = lane >> 3, kg = lane & 7;
        const float* a = mA + ((size_t)hh * 16 + ti * 4) * PD;
        const float* b = mB + ((size_t)hh * 16 + tj * 4) * PD;
        float acc[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) acc[i] = 0.f;
        for (int e = kg * 4; e < PD; e += 32) {
            float4 x[4], y[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                x[i] = *reinterpret_cast<const float4*>(a + (size_t)i * PD + e);
                y[i] = *reinterpret_cast<const float4*>(b + (size_t)i * PD + e);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    float s = acc[i * 4 + j];
                    s = fmaf(x[i].x, y[j].x, s); s = fmaf(x[i].y, y[j].y, s);
                    s = fmaf(x[i].z, y[j].z, s); s = fmaf(x[i].w, y[j].w, s);
                    acc[i * 4 + j] = s;
                }
        }
        // the eight lanes' sums: every exchange halves the values that a lane still carries
        int first = 0;
#pragma unroll
        for (int s = 0; s < 3; ++s) {
            const int half = 8 >> s;
            const bool up = lane & (1 << s);
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (i < half) {
                    const float keep = up ? acc[i + half] : acc[i], give = up ? acc[i] : acc[i + half];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << s);
                }
            first += up ? half : 0;
        }
        float* dst = gm + hh * 256 + (ti * 4 + (first >> 2)) * 16 + tj * 4 + (first & 3);
        dst[0] = acc[0];
        dst[1] = acc[1];
    }
    __syncthreads();
    auto row8 = [](const float* p, float (&x)[DL_TOK]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    };
    // forward substitution, a thread a channel; behind the channels eight columns a head for M and N
    float* out = rec + ((size_t)item * H + h0) * (33 * (size_t)DP + 128);
    const size_t rs = 33 * (size_t)DP + 128;
#pragma unroll
    for (int q = 0; q < NC; ++q) {
        const int ch = tid + 256 * q;
        if (ch < nh * D) {
            const int hh = ch / D, e = ch - hh * D;
            const float* g = gm + hh * 256;
            const float* a = mA + (size_t)hh * 16 * PD + e;
            float* o = out + hh * rs + e;
            const float last = w[q][DL_TOK - 1];
            float kt[DL_TOK];
#pragma unroll
            for (int i = 0; i < DL_TOK; ++i) {
                float s = a[i * PD], t = r[q][i], gr[DL_TOK], gq[DL_TOK];
                row8(g + i * 16 + 8, gr);
                row8(g + (8 + i) * 16 + 8, gq);
#pragma unroll
                for (int j = 0; j < i; ++j) s = fmaf(-gr[j], kt[j], s);
                kt[i] = s;
#pragma unroll
                for (int j = 0; j <= i; ++j) t = fmaf(-gq[j], kt[j], t);
                o[(size_t)i * DP] = s;
                o[(size_t)(8 + i) * DP] = t;
                o[(size_t)(16 + i) * DP] = k[q][i] * last;
                o[(size_t)(24 + i) * DP] = -(z[q][i] * last);
            }
            o[(size_t)32 * DP] = last;
        }
    }
    for (int u = tid; u < nh * 8; u += 256) {
        const int hh = u >> 3, c = u & 7;
        const float* g = gm + hh * 256;
        float* o = out + hh * rs + 33 * (size_t)DP + c;
        float m[DL_TOK];
#pragma unroll
        for (int i = 0; i < DL_TOK; ++i) {
            float s = c < i ? g[i * 16 + c] : 0.f, t = c <= i ? g[(8 + i) * 16 + c] : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) s = fmaf(-g[i * 16 + 8 + j], m[j], s);
            m[i] = s;
#pragma unroll
            for (int j = 0; j <= i; ++j) t = fmaf(-g[(8 + i) * 16 + 8 + j], m[j], t);
            o[i * 8] = s;
            o[64 + i * 8] = t;
        }
    }
    if (DP != D)
        for (int i = tid; i < nh * 33 * (DP - D); i += 256) {
            const int row = i / (DP - D), hh = row / 33;
            out[hh * rs + (size_t)(row - hh * 33) * DP + D + i % (DP - D)] = 0.f;
        }
    // the recurrence has few, long-lived blocks: begun while these blocks fill the SMs they would pile up on whichever
    // SMs have room first
    pdl_launch_dependents();
}

// proj: float [T][ld], rows [r | k | v | z | g | x]; the step's n_items blocks of up to eight tokens (item_seq: the request, item_idx:
// the block's number in it); rec: float [n_items][H][33 pad(D) + 128].
ACV_API int acv_delta_blocks(const float* proj, int ld, const float* w2t, const float* w0, const int* item_seq,
                             const int* item_idx, const int* cu_q, float* rec, int n_items, int H, int D, int L,
                             cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (H <= 0 || D <= 0 || D > 512 || L <= 0 || L > 1024 || ld < 5 * H * D + L) return ACV_ERR_SIZE;
    int heads = 256 / D;
    heads = heads < 1 ? 1 : (heads > 32 ? 32 : heads);
    if (heads > H) heads = H;
    const int PD = (D + 3) & ~3;
    const size_t smem = ((size_t)L * DL_TOK + (size_t)heads * (32 * PD + 256 + DL_TOK)) * sizeof(float);
    const dim3 grid(n_items, (H + heads - 1) / heads);
    if (grid.y > 65535 || smem > 200 * 1024) return ACV_ERR_SIZE;
#define DB_LAUNCH(N)                                                                                                          \
    do {                                                                                                                      \
        static AcvSmemConfig cfg;                                                                                             \
        if (smem > 48 * 1024)                                                                                                 \
            if (int e = acv_ensure_smem(cfg, delta_blocks_kernel<N>, (int)smem)) return e;                                    \
        acv_launch(PDL_MISC, delta_blocks_kernel<N>, grid, 256, smem, stream, proj, ld, w2t, w0, item_seq, item_idx, cu_q,    \
                   rec, H, D, delta_pad(D), L, heads);                                                                        \
    } while (0)
    if (D <= 256) DB_LAUNCH(1);
    else DB_LAUNCH(2);
#undef DB_LAUNCH
    return acv_launch_status();
}

ACV_API int acv_delta_record_floats(int D) { return (int)delta_record(delta_pad(D)); }

// ----------------------------------------------------------------------------- the recurrence
// Columns of S are recurrences of their own.  A thread keeps R rows of C neighbouring columns in registers (pairs of rows,
// two to an instruction), G lanes share a column, a block's NW warps hold NW * 32 / G * C columns and walk the request's
// blocks of eight tokens; records and values are copied asynchronously, STAGES - 1 blocks ahead.
typedef unsigned long long f2;              // two floats that one instruction works on
__device__ __forceinline__ f2 f2_pack(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void f2_split(f2 x, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(x)); }
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

// The sums over the G lanes of a column of eight values each, one for every token of the block.  A lane keeps token i ^ m in
// v[i], m = first_of(lane): the half that it gives away at an exchange is then the half that its partner keeps, and an
// exchange halves what a lane still carries (7 exchanges at G = 8).  Afterwards v[0 .. LEFT) are the totals of the tokens
// m + i, LEFT = G >= 8 ? 1 : 8 / G.
template <int G>
__device__ __forceinline__ void lanes_sum8(float (&v)[8]) {
    if constexpr (G > 1)
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] += __shfl_xor_sync(0xffffffffu, v[i + 4], 1);
    if constexpr (G > 2)
#pragma unroll
        for (int i = 0; i < 2; ++i) v[i] += __shfl_xor_sync(0xffffffffu, v[i + 2], 2);
    if constexpr (G > 4) v[0] += __shfl_xor_sync(0xffffffffu, v[1], 4);
#pragma unroll
    for (int o = 8; o < G; o <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
}
template <int G>
__device__ __forceinline__ int first_of(int lane) {
    return (G > 1 ? (lane & 1) * 4 : 0) + (G > 2 ? (lane & 2) : 0) + (G > 4 ? (lane & 4) >> 2 : 0);
}
// the lane (within its column's G) and the place at which token e's total lies
template <int G>
__device__ __forceinline__ constexpr int lane_of(int e) {
    return (G > 1 ? (e >> 2) & 1 : 0) | (G > 2 ? ((e >> 1) & 1) << 1 : 0) | (G > 4 ? (e & 1) << 2 : 0);
}
template <int G>
__device__ __forceinline__ constexpr int place_of(int e) { return G >= 8 ? 0 : e & (8 / G - 1); }

// KD: a record as above, state [D, D].  Without it the record is that of a gated delta rule, [kt' 8][rt 8][k' 8] rows, M, N and
// the block's decay (one number, padded to four), and the state is [D, DV]:  u = kt' S + M v,  o = rt S + N v,
// S_8 = decay S + sum_j k'_j u_j^T.
template <int R, int G, int C, int NW, int STAGES, bool KD>
__global__ void __launch_bounds__(NW * 32)
delta_kernel(const float* __restrict__ rec, const float* __restrict__ values, int ld, float* __restrict__ state,
             const int* __restrict__ slots, const int* __restrict__ cu_q, const int* __restrict__ first_block,
             float* __restrict__ o, int H, int D, int DV, int vec) {
    constexpr int DP = R * G, DVT = NW * (32 / G) * C, R2 = R / 2, LEFT = G >= 8 ? 1 : 8 / G;
    constexpr int PF = R < 4 ? 1 : 2;       // pairs in a piece that one load brings
    constexpr int REC = KD ? 33 * DP + 128 : 24 * DP + 132, MATS = (KD ? 33 : 24) * DP, SET = REC + 8 * DVT, NT = NW * 32;
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * DVT;
    const int t0 = cu_q[seq], t1 = cu_q[seq + 1];
    if (t1 <= t0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane % G, cl = (warp * (32 / G) + lane / G) * C, c = c0 + cl;
    const int I = H * DV, nb = (t1 - t0 + 7) >> 3;
    const int e0 = first_of<G>(lane);
    float* st = state + ((size_t)slots[seq] * H + h) * D * DV;
    const float* recs = rec + ((size_t)first_block[seq] * H + h) * REC;
    const float* vals = values + (size_t)t0 * ld + (size_t)h * DV + c0;

    auto stage = [&](int b) {
        float* s = sm + (b % STAGES) * SET;
        const float* src = recs + (size_t)b * H * REC;
        for (int i = tid * 4; i < REC; i += NT * 4) cp_async16(smem_u32(s + i), src + i, true);
        float* vs = s + REC;
        if (vec) {
            for (int i = tid * 4; i < 8 * DVT; i += NT * 4) {
                const int tt = i / DVT, e = i % DVT, t = b * 8 + tt;
                const bool in = t < t1 - t0 && c0 + e < DV;
                cp_async16(smem_u32(vs + i), in ? (const void*)(vals + (size_t)t * ld + e) : (const void*)values, in);
            }
        } else {
            for (int i = tid; i < 8 * DVT; i += NT) {
                const int tt = i / DVT, e = i % DVT, t = b * 8 + tt;
                vs[i] = t < t1 - t0 && c0 + e < DV ? vals[(size_t)t * ld + e] : 0.f;
            }
        }
    };
    // a thread's rows: pairs of neighbours, PF pairs to a piece, pieces G apart
    f2 S[C][R2];
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < R2; ++i) {
            const int d = ((i / PF) * G + g) * PF * 2 + (i % PF) * 2;
            const bool in = c + j < DV;
            S[j][i] = f2_pack(in && d < D ? st[(size_t)d * DV + c + j] : 0.f, in && d + 1 < D ? st[(size_t)(d + 1) * DV + c + j] : 0.f);
        }
#pragma unroll
    for (int b = 0; b < STAGES - 1; ++b) {
        if (b < nb) stage(b);
        cp_async_commit();
    }
    auto rows = [&](const float* row, f2 (&x)[R2]) {
#pragma unroll
        for (int i = 0; i < R2; i += PF) {
            if constexpr (PF == 2) {
                const ulonglong2 q = reinterpret_cast<const ulonglong2*>(row)[(i >> 1) * G + g];
                x[i] = q.x; x[i + 1] = q.y;
            } else {
                x[i] = reinterpret_cast<const f2*>(row)[i * G + g];
            }
        }
    };
    auto dot = [&](const f2 (&x)[R2], const f2 (&y)[R2]) {
        f2 a = f2_mul(x[0], y[0]);
#pragma unroll
        for (int i = 1; i < R2; ++i) a = f2_fma(x[i], y[i], a);
        float lo, hi;
        f2_split(a, lo, hi);
        return lo + hi;
    };
    for (int b = 0; b < nb; ++b) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();                    // block b is there; everyone is done with block b - 1, whose buffer is filled next
        if (b + STAGES - 1 < nb) stage(b + STAGES - 1);
        cp_async_commit();
        const float* s = sm + (b % STAGES) * SET;
        const float* mn = s + MATS;
        const float* vs = s + REC + cl;
        float y[C][8], z[C][8], v[C][8];
        f2 x[R2];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            rows(s + (i ^ e0) * DP, x);
#pragma unroll
            for (int j = 0; j < C; ++j) y[j][i] = dot(x, S[j]);
        }
#pragma unroll
        for (int j = 0; j < C; ++j) lanes_sum8<G>(y[j]);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            rows(s + (8 + (i ^ e0)) * DP, x);
#pragma unroll
            for (int j = 0; j < C; ++j) z[j][i] = dot(x, S[j]);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < C; ++j) v[j][i] = vs[i * DVT + j];
        // this lane's tokens: p (its sum over the values of the tokens before it; the new values u without KD), later o
#pragma unroll
        for (int l = 0; l < LEFT; ++l) {
            const float4 m0 = *reinterpret_cast<const float4*>(mn + (e0 + l) * 8), m1 = *reinterpret_cast<const float4*>(mn + (e0 + l) * 8 + 4);
#pragma unroll
            for (int j = 0; j < C; ++j) {
                float a = fmaf(m0.x, v[j][0], y[j][l]), d = m0.y * v[j][1];
                a = fmaf(m0.z, v[j][2], a); d = fmaf(m0.w, v[j][3], d);
                a = fmaf(m1.x, v[j][4], a); d = fmaf(m1.y, v[j][5], d);
                if constexpr (!KD) d = fmaf(m1.w, v[j][7], d);     // (with KD a token's p holds no value of its own)
                y[j][l] = fmaf(m1.z, v[j][6], a) + d;
            }
        }
        if constexpr (KD) {
            rows(s + 32 * DP, x);
        } else {
            const float decay = mn[128];
#pragma unroll
            for (int i = 0; i < R2; ++i) x[i] = f2_pack(decay, decay);
        }
#pragma unroll
        for (int j = 0; j < C; ++j)
#pragma unroll
            for (int i = 0; i < R2; ++i) S[j][i] = f2_mul(x[i], S[j][i]);
        if constexpr (KD) {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                rows(s + (16 + i) * DP, x);
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const f2 vv = f2_pack(v[j][i], v[j][i]);
#pragma unroll
                    for (int q = 0; q < R2; ++q) S[j][q] = f2_fma(x[q], vv, S[j][q]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            rows(s + ((KD ? 24 : 16) + i) * DP, x);
#pragma unroll
            for (int j = 0; j < C; ++j) {
                const float p = G > 1 ? __shfl_sync(0xffffffffu, y[j][place_of<G>(i)], lane_of<G>(i), G) : y[j][i];
                const f2 pp = f2_pack(p, p);
#pragma unroll
                for (int q = 0; q < R2; ++q) S[j][q] = f2_fma(x[q], pp, S[j][q]);
            }
        }
#pragma unroll
        for (int j = 0; j < C; ++j) lanes_sum8<G>(z[j]);
        if (G <= 8 || g < 8) {
#pragma unroll
            for (int l = 0; l < LEFT; ++l) {
                const float4 m0 = *reinterpret_cast<const float4*>(mn + 64 + (e0 + l) * 8), m1 = *reinterpret_cast<const float4*>(mn + 64 + (e0 + l) * 8 + 4);
                const int t = t0 + b * 8 + e0 + l;
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    float a = fmaf(m0.x, v[j][0], z[j][l]), d = m0.y * v[j][1];
                    a = fmaf(m0.z, v[j][2], a); d = fmaf(m0.w, v[j][3], d);
                    a = fmaf(m1.x, v[j][4], a); d = fmaf(m1.y, v[j][5], d);
                    a = fmaf(m1.z, v[j][6], a); d = fmaf(m1.w, v[j][7], d);
                    if (t < t1 && c + j < DV) o[(size_t)t * I + (size_t)h * DV + c + j] = a + d;
                }
            }
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < R2; ++i) {
            const int d = ((i / PF) * G + g) * PF * 2 + (i % PF) * 2;
            float a, b;
            f2_split(S[j][i], a, b);
            if (c + j < DV && d < D) st[(size_t)d * DV + c + j] = a;
            if (c + j < DV && d + 1 < D) st[(size_t)(d + 1) * DV + c + j] = b;
        }
}

template <int R, int G, int C, int NW, int STAGES, bool KD>
static int launch_delta(const float* rec, const float* values, int ld, float* state, const int* slots, const int* cu_q,
                        const int* first_block, float* o, int n_seqs, int H, int D, int DV, cudaStream_t stream) {
    constexpr int DVT = NW * (32 / G) * C;
    constexpr size_t smem = (size_t)STAGES * ((KD ? 33 * R * G + 128 : 24 * R * G + 132) + 8 * DVT) * sizeof(float);
    static_assert(smem <= 227 * 1024 && DVT % 4 == 0, "a block's stages fit, values come in 16-byte pieces");
    static AcvSmemConfig cfg;
    if (smem > 48 * 1024)
        if (int e = acv_ensure_smem(cfg, delta_kernel<R, G, C, NW, STAGES, KD>, (int)smem)) return e;
    const int vec = DV % 4 == 0 && ld % 4 == 0 && !((uintptr_t)values & 15);
    const dim3 grid(n_seqs, H, (DV + DVT - 1) / DVT);
    if (grid.y > 65535 || grid.z > 65535) return ACV_ERR_SIZE;
    acv_launch(PDL_ATTN, delta_kernel<R, G, C, NW, STAGES, KD>, grid, NW * 32, smem, stream, rec, values, ld, state, slots, cu_q,
               first_block, o, H, D, DV, vec);
    return acv_launch_status();
}

template <bool KD>
static int delta_by_size(const float* rec, const float* values, int ld, float* state, const int* slots, const int* cu_q,
                         const int* first_block, float* o, int n_seqs, int H, int D, int DV, int form, cudaStream_t stream) {
#define DL_CASE(RR, GG, CC, WW, SS) \
    return launch_delta<RR, GG, CC, WW, SS, KD>(rec, values, ld, state, slots, cu_q, first_block, o, n_seqs, H, D, DV, stream);
    if (D <= 8) DL_CASE(8, 1, 1, 1, 3)
    if (D <= 16) DL_CASE(8, 2, 1, 1, 3)
    if (D <= 32) DL_CASE(8, 4, 1, 4, 3)
    // few columns for the device: four warps to sixteen columns; more: two warps, then one (fewer instructions a column)
    const long long tiles = (long long)n_seqs * H * ((DV + 15) / 16);
    if constexpr (!KD) {        // (shorter records: measured to want their own shapes)
        if (D > 32 && D <= 128 && !form) form = tiles <= 180 ? 1 : tiles <= 600 ? 2 : 3;
        if (D > 32 && D <= 64) {
            if (form == 1) DL_CASE(8, 8, 2, 2, 4)
            if (form == 2) DL_CASE(4, 16, 4, 2, 4)
            DL_CASE(8, 8, 4, 1, 3)
        }
        if (D > 64 && D <= 128) {
            if (form == 1) DL_CASE(8, 16, 2, 4, 4)
            if (form == 2) DL_CASE(8, 16, 4, 2, 3)
            DL_CASE(16, 8, 4, 2, 4)
        }
    }
    if (D <= 64) {
        if (!form) form = tiles <= 180 ? 1 : tiles <= 600 ? 2 : 3;
        if (form == 1) DL_CASE(4, 16, 2, 4, 3)
        if (form == 2) DL_CASE(4, 16, 4, 2, 3)
        DL_CASE(8, 8, 4, 1, 3)
    }
    if (D <= 128) {
        if (!form) form = tiles <= 600 ? 1 : 2;
        if (form == 1) DL_CASE(8, 16, 2, 4, 3)
        DL_CASE(8, 16, 4, 2, 3)
    }
    if (D <= 256) DL_CASE(8, 32, 1, 4, 3)
    DL_CASE(16, 32, 1, 4, 2)
#undef DL_CASE
}

// After acv_delta_blocks, or with `gated` after acv_gated_delta_blocks.  values: rows of `ld` floats whose first H*DV columns are
// the values (DV = D unless gated); first_block: the number of each request's first block among the step's items; o: float
// [T][H*DV]; state: float [slots][H][D][DV]; key heads of up to 512 channels.  form: 0, or a choice among the shapes of a
// block (timing).
ACV_API int acv_delta(const float* rec, const float* values, int ld, float* state, const int* slots, const int* cu_q,
                      const int* first_block, float* o, int n_seqs, int H, int D, int DV, int gated, int form,
                      cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || D <= 0 || D > 512 || DV <= 0 || (!gated && DV != D)) return ACV_ERR_SIZE;
    if ((uintptr_t)rec & 15) return ACV_ERR_ALIGN;
    return gated ? delta_by_size<false>(rec, values, ld, state, slots, cu_q, first_block, o, n_seqs, H, D, DV, form, stream)
                 : delta_by_size<true>(rec, values, ld, state, slots, cu_q, first_block, o, n_seqs, H, D, DV, form, stream);
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
