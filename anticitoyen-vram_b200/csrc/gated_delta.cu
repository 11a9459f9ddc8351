// A gated delta rule: one decay and one step size per head and token, keys and queries shared by groups of heads, with a short
// causal convolution in front.
//
// A token's row of the input product is [q | k | v | z | b | a]: q, k of G heads of D channels, v and the output gate z of H
// heads of DV, the step size b and the decay a of every head.  All float.  Per (request, head h), with the q and k of head
// h / (H/G), y = silu(conv(.)) of q, k and v over the request's tokens (K taps a channel, the last one the current token's),
//
//     k <- y_k / sqrt(sum(y_k^2) + 1e-6),    q <- y_q / sqrt(sum(y_q^2) + 1e-6) / sqrt(D),    v <- y_v
//     beta = sigmoid(b),    g = exp(-rate_h softplus(a + shift_h))
//     S <- g S;    u = beta (v - S^T k);    S <- S + k u^T;    o = S^T q                       S: [D, DV] float, zero at first
//
//   acv_gated_delta_blocks   everything that does not need the state, for eight tokens of a request at a time
//   acv_delta (gated)        the recurrence over those blocks (csrc/general_delta.cu), o float
//   acv_gated_delta_step     steps in which every request brings one token: all of the above, the head's norm, weight and gate
//                            in one launch
//
// Eight tokens at once: with R_ij = g_{j+1} .. g_i (products of decays only: nothing is divided by, so decays of any size are
// safe), c_i = g_1 .. g_i, and the state S in front of the block,
//
//     A_ij = beta_i R_ij <k_i, k_j> (j < i)      Q_ij = R_ij <q_i, k_j> (j <= i)      M = (I + A)^-1 diag(beta)      N = Q M
//     u = M v - M diag(c) k S           o = diag(c) q S + N v - N diag(c) k S           S_8 = c_8 S + sum_j R_8j k_j u_j^T
//
// A block's record (floats, channels padded to DP with zeros): -M diag(c) k [8][DP], diag(c) q - N diag(c) k [8][DP],
// R_8j k_j [8][DP], M [8][8], N [8][8], c_8 and three zeros.  Tokens behind a portion's end are k = q = 0, g = 1, beta = 0.
//
// What the convolution keeps of a request: the rows of its last inputs in a ring of K rows, position p in row p mod K (a step
// of one token reads K - 1 rows and writes the one that none of its readers reads).
#include "mma_tiles.cuh"

#define GD_TOK 8
#define GD_UNIT_EPS 1e-6f
#define GD_CHANNELS 256         // query channels of a thread block of the blocks' kernel, where heads are small enough

static int gated_delta_pad(int D) {
    int p = 8;
    while (p < D) p <<= 1;
    return p;
}

__device__ __forceinline__ float gd_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float gd_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gd_decay(float a, float rate, float shift) { return expf(-rate * gd_softplus(a + shift)); }

// The convolution of one channel at eight tokens.  x: the channel at the first of them (rows of ld), `off` tokens of the portion lie
// in front of it, `pos` is its position, n of the eight exist; w: the channel's taps, rows of C; ring: the channel's kept
// inputs, rows of C.  KT > 0: K <= KT, the inputs wait in registers.
template <int KT>
__device__ __forceinline__ void conv8(const float* __restrict__ x, int ld, const float* __restrict__ w, int C, int K,
                                      const float* ring, int off, int pos, int n, float (&y)[GD_TOK]) {
    auto input = [&](int rho) {         // rho: relative to the first token
        if (rho >= n) return 0.f;
        if (rho >= -off) return x[(ptrdiff_t)rho * ld];
        return pos + rho >= 0 ? ring[(size_t)((pos + rho) % K) * C] : 0.f;
    };
    if constexpr (KT > 0) {
        float in[KT - 1 + GD_TOK], tap[KT];
#pragma unroll
        for (int i = 0; i < KT - 1 + GD_TOK; ++i) in[i] = i - (KT - 1) > -K ? input(i - (KT - 1)) : 0.f;
#pragma unroll
        for (int j = 0; j < KT; ++j) tap[j] = j < K ? w[(size_t)(K - 1 - j) * C] : 0.f;
#pragma unroll
        for (int t = 0; t < GD_TOK; ++t) {
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < KT; ++j) s = fmaf(tap[j], in[t + KT - 1 - j], s);
            y[t] = s;
        }
    } else {
#pragma unroll
        for (int t = 0; t < GD_TOK; ++t) y[t] = 0.f;
        for (int j = 0; j < K; ++j) {
            const float tap = w[(size_t)(K - 1 - j) * C];
#pragma unroll
            for (int t = 0; t < GD_TOK; ++t) y[t] = fmaf(tap, input(t - j), y[t]);
        }
    }
}

// the last K - 1 inputs of a portion (rows first .. first + len of proj, the first at position pos) into the ring, one channel
__device__ __forceinline__ void keep_inputs(const float* __restrict__ x, int ld, float* ring, int C, int K, int len, int pos) {
    for (int i = max(0, len - (K - 1)); i < len; ++i) ring[(size_t)((pos + i) % K) * C] = x[(size_t)i * ld];
}

// ----------------------------------------------------------------------------- the blocks' records
// grid (blocks of tokens, tiles of `ng` q/k heads); the heads that read them belong to a thread block, and so do their channels
// of the convolution.
template <int KT>
__global__ void __launch_bounds__(256)
gated_delta_blocks_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ wt, const float* __restrict__ rate,
                          const float* __restrict__ shift, float* ring, const int* __restrict__ slots,
                          const int* __restrict__ positions, const int* __restrict__ item_seq, const int* __restrict__ item_idx,
                          const int* __restrict__ cu_q, float* __restrict__ values, float* __restrict__ rec, int G, int H,
                          int D, int DV, int DP, int K, int ng) {
    extern __shared__ __align__(16) float sm[];
    const int PD = (D + 3) & ~3, r = H / G;
    float* rows = sm;                       // [ng][16][PD]: y_q of the eight tokens, y_k
    float* gram = rows + (size_t)ng * 16 * PD;      // [ng][144]: <q, k> [8][8], <k, k> [8][8], what brings y_q, y_k to their length [16]
    float* wa = gram + ng * 144;            // [8 warps][128]: A, Q of the head that a warp is at
    float* coef = wa + 8 * 128;             // [ng r][144]
    pdl_wait();
    const int item = blockIdx.x, g0 = blockIdx.y * ng, gn = min(ng, G - g0), hn = gn * r, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = item_seq[item], idx = item_idx[item];
    const int first = cu_q[seq], off = idx * GD_TOK, t0 = first + off, len = cu_q[seq + 1] - first;
    const int n = min(GD_TOK, len - off), pos = positions[t0];
    const int C = 2 * G * D + H * DV, I = H * DV;
    float* slot = ring + (size_t)slots[seq] * K * C;
    const float* base = proj + (size_t)t0 * ld;
    for (int ch = tid; ch < 2 * gn * D; ch += 256) {
        const bool is_k = ch >= gn * D;
        const int at = is_k ? ch - gn * D : ch, gl = at / D, e = at - gl * D, c = (is_k ? G * D : 0) + g0 * D + at;
        float y[GD_TOK];
        conv8<KT>(base + c, ld, wt + c, C, K, slot + c, off, pos, n, y);
#pragma unroll
        for (int t = 0; t < GD_TOK; ++t) rows[(size_t)(gl * 16 + (is_k ? 8 : 0) + t) * PD + e] = t < n ? gd_silu(y[t]) : 0.f;
    }
    for (int ch = tid; ch < hn * DV; ch += 256) {
        const int at = g0 * r * DV + ch, c = 2 * G * D + at;
        float y[GD_TOK];
        conv8<KT>(base + c, ld, wt + c, C, K, slot + c, off, pos, n, y);
#pragma unroll
        for (int t = 0; t < GD_TOK; ++t)
            if (t < n) values[(size_t)(t0 + t) * I + at] = gd_silu(y[t]);
    }
    __syncthreads();
    if (idx == 0 && K > 1 && K <= GD_TOK + 1) {     // no other block reads these channels' kept inputs (off >= K - 1 there)
        const float* p = proj + (size_t)first * ld;
        const int w = gn * D;
        for (int ch = tid; ch < 2 * w + hn * DV; ch += 256) {
            const int c = ch < w ? g0 * D + ch : ch < 2 * w ? G * D + g0 * D + ch - w : 2 * G * D + g0 * r * DV + ch - 2 * w;
            keep_inputs(p + c, ld, slot + c, C, K, len, pos);
        }
    }
    // a warp one token's row of both matrices
    for (int u = warp; u < gn * 8; u += 8) {
        const int gl = u >> 3, i = u & 7;
        const float* base_q = rows + (size_t)gl * 16 * PD;
        const float* base_k = base_q + (size_t)8 * PD;
        float a[8], b[8], qq = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] = b[j] = 0.f;
        for (int e = lane; e < D; e += 32) {
            const float qe = base_q[(size_t)i * PD + e], ke = base_k[(size_t)i * PD + e];
            qq = fmaf(qe, qe, qq);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float kj = base_k[(size_t)j * PD + e];
                a[j] = fmaf(qe, kj, a[j]);
                b[j] = fmaf(ke, kj, b[j]);
            }
        }
        // both rows' sixteen sums over the lanes: every exchange halves the values that a lane still carries
        const bool up4 = lane & 16, up3 = lane & 8, up2 = lane & 4, up1 = lane & 2;
        float x[8], y[4], z[2];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = (up4 ? b[j] : a[j]) + __shfl_xor_sync(0xffffffffu, up4 ? a[j] : b[j], 16);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = (up3 ? x[j + 4] : x[j]) + __shfl_xor_sync(0xffffffffu, up3 ? x[j] : x[j + 4], 8);
#pragma unroll
        for (int j = 0; j < 2; ++j) z[j] = (up2 ? y[j + 2] : y[j]) + __shfl_xor_sync(0xffffffffu, up2 ? y[j] : y[j + 2], 4);
        float sum = (up1 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, up1 ? z[0] : z[1], 2);
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        qq = warp_sum(qq);
        float* gm = gram + gl * 144;
        const int j = (up3 ? 4 : 0) + (up2 ? 2 : 0) + (up1 ? 1 : 0);
        if (!(lane & 1)) gm[(up4 ? 64 : 0) + i * 8 + j] = sum;
        if (lane == 0) gm[128 + i] = 1.f / (sqrtf(qq + GD_UNIT_EPS) * sqrtf((float)D));
        if (up4 && j == i && !(lane & 1)) gm[136 + i] = 1.f / sqrtf(sum + GD_UNIT_EPS);
    }
    __syncthreads();
    const size_t rs = 24 * (size_t)DP + 132;
    float* out = rec + ((size_t)item * H + (size_t)g0 * r) * rs;
    // a warp a head; lane j (mod 8) owns column j
    for (int hh = warp; hh < hn; hh += 8) {
        const int h = g0 * r + hh, j = lane & 7;
        const float* qk = gram + hh / r * 144;
        const float* kk = qk + 64;
        const float* inv = qk + 128;
        float beta = 0.f, g = 1.f;
        if (j < n) {
            const float* row = base + (size_t)j * ld + C + I;
            beta = gd_sigmoid(row[h]);
            g = gd_decay(row[H + h], rate[h], shift[h]);
        }
        float* A = wa + warp * 128;
        float* Q = A + 64;
        float* cf = coef + hh * 144;
        float bi[8], c = 1.f, run = 1.f, mine = 1.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            bi[i] = __shfl_sync(0xffffffffu, beta, i);
            const float gi = __shfl_sync(0xffffffffu, g, i);
            c *= gi;
            if (i == j) mine = c;
            if (i > j) run *= gi;
            if (lane < 8) {
                A[i * 8 + j] = i > j ? bi[i] * run * (kk[i * 8 + j] * inv[8 + i] * inv[8 + j]) : 0.f;
                Q[i * 8 + j] = i >= j ? run * (qk[i * 8 + j] * inv[i] * inv[8 + j]) : 0.f;
            }
        }
        __syncwarp();
        if (lane < 8) {
            float m[8];
            float* mats = out + hh * rs + 24 * (size_t)DP;
            const float scale = mine * inv[8 + j];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                float s = i == j ? bi[i] : 0.f, t = 0.f;
#pragma unroll
                for (int l = 0; l < i; ++l) s = fmaf(-A[i * 8 + l], m[l], s);
                m[i] = s;
#pragma unroll
                for (int l = 0; l <= i; ++l) t = fmaf(Q[i * 8 + l], m[l], t);
                mats[i * 8 + j] = s;
                mats[64 + i * 8 + j] = t;
                cf[i * 8 + j] = -s * scale;
                cf[64 + i * 8 + j] = -t * scale;
            }
            cf[128 + j] = mine * inv[j];
            cf[136 + j] = run * inv[8 + j];
            if (j < 4) mats[128 + j] = j == 0 ? c : 0.f;
        }
        __syncwarp();
    }
    __syncthreads();
    auto row8 = [](const float* p, float (&x)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    };
    for (int u = tid; u < hn * DP; u += 256) {
        const int hh = u / DP, e = u - hh * DP;
        const float* mine = rows + (size_t)(hh / r) * 16 * PD + e;
        float* o = out + hh * rs + e;
        if (e >= D) {
#pragma unroll
            for (int i = 0; i < 24; ++i) o[(size_t)i * DP] = 0.f;
            continue;
        }
        const float* cf = coef + hh * 144;
        float k[8], x[8], gam[8], dec[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) k[i] = mine[(size_t)(8 + i) * PD];
        row8(cf + 128, gam);
        row8(cf + 136, dec);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float s = 0.f, t = gam[i] * mine[(size_t)i * PD];
            row8(cf + i * 8, x);
#pragma unroll
            for (int l = 0; l <= i; ++l) s = fmaf(x[l], k[l], s);
            row8(cf + 64 + i * 8, x);
#pragma unroll
            for (int l = 0; l <= i; ++l) t = fmaf(x[l], k[l], t);
            o[(size_t)i * DP] = s;
            o[(size_t)(8 + i) * DP] = t;
            o[(size_t)(16 + i) * DP] = dec[i] * k[i];
        }
    }
    pdl_launch_dependents();
}

// more taps than a block of tokens reaches back: the kept inputs are replaced once every block has read them
__global__ void gated_delta_keep_kernel(const float* __restrict__ proj, int ld, float* ring, const int* __restrict__ slots,
                                        const int* __restrict__ positions, const int* __restrict__ cu_q, int C, int K) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    const int first = cu_q[seq], len = cu_q[seq + 1] - first;
    if (c >= C || len <= 0) return;
    keep_inputs(proj + (size_t)first * ld + c, ld, ring + (size_t)slots[seq] * K * C + c, C, K, len, positions[first]);
}

ACV_API int acv_gated_delta_record_floats(int D) { return 24 * gated_delta_pad(D) + 132; }

// proj: float [T][ld], rows [q | k | v | z | b | a]; wt: float [K][2 G D + H DV], the taps transposed; rate, shift: float [H];
// ring: float [slots][K][2 G D + H DV]; the step's n_items blocks of up to eight tokens (item_seq, item_idx as for
// acv_delta_blocks); values: float [T][H DV]; rec: float [n_items][H][record].
ACV_API int acv_gated_delta_blocks(const float* proj, int ld, const float* wt, const float* rate, const float* shift, float* ring,
                                   const int* slots, const int* positions, const int* item_seq, const int* item_idx,
                                   const int* cu_q, float* values, float* rec, int n_items, int n_seqs, int G, int H, int D,
                                   int DV, int K, cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (G <= 0 || G > 65535 || H <= 0 || H % G || D <= 0 || D > 512 || DV <= 0 || K < 1 || ld < 2 * G * D + 2 * H * DV + 2 * H)
        return ACV_ERR_SIZE;
    const int PD = (D + 3) & ~3, C = 2 * G * D + H * DV;
    // q/k heads of a thread block: enough for its threads, and for its warps where a warp makes a head's matrices
    auto bytes = [&](int n) { return (8 * 128 + (size_t)n * (16 * PD + 144 + (size_t)(H / G) * 144)) * sizeof(float); };
    int ng = 1;
    while (ng * 2 <= G && ng * 2 * D <= GD_CHANNELS && bytes(ng * 2) <= 64 * 1024) ng *= 2;
    const size_t smem = bytes(ng);
    if (smem > 200 * 1024) return ACV_ERR_SIZE;
    const dim3 grid(n_items, (G + ng - 1) / ng);
#define GB_LAUNCH(N)                                                                                                          \
    do {                                                                                                                      \
        static AcvSmemConfig cfg;                                                                                             \
        if (smem > 48 * 1024)                                                                                                 \
            if (int e = acv_ensure_smem(cfg, gated_delta_blocks_kernel<N>, (int)smem)) return e;                              \
        acv_launch(PDL_MISC, gated_delta_blocks_kernel<N>, grid, 256, smem, stream, proj, ld, wt, rate, shift, ring, slots,   \
                   positions, item_seq, item_idx, cu_q, values, rec, G, H, D, DV, gated_delta_pad(D), K, ng);                 \
    } while (0)
    if (K <= 4) GB_LAUNCH(4);
    else GB_LAUNCH(0);
#undef GB_LAUNCH
    if (K > GD_TOK + 1)
        acv_launch(PDL_MISC, gated_delta_keep_kernel, dim3(n_seqs, (C + 255) / 256), 256, 0, stream, proj, ld, ring, slots,
                   positions, cu_q, C, K);
    return acv_launch_status();
}

// ----------------------------------------------------------------------------- one token a request, everything
// A block of 256 threads a (request, head).  A thread holds RPT rows of four neighbouring columns: c4 = DV / 4 threads cover a
// row, NG = 256 / c4 groups of rows stand side by side; sums over rows pass through shared memory.  What the block needs beside
// the state is asked for in front of it and all at once (FEW: up to four taps and two channels of the convolution a thread),
// so that no chain of loads stands between the state's arrival and its way back.
template <typename T, int RPT, bool FEW>
__global__ void __launch_bounds__(256, RPT <= 16 ? 2 : 1)
gated_delta_step_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ wt, const float* __restrict__ rate,
                        const float* __restrict__ shift, const float* __restrict__ weight, float eps, float* ring,
                        const int* __restrict__ ring_slots, float* __restrict__ state, const int* __restrict__ slots,
                        const int* __restrict__ positions, const int* __restrict__ cu_q, T* __restrict__ out, int ldo, int G,
                        int H, int D, int DV, int K) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    const int D4 = (D + 3) & ~3;
    float* vs = sm;                         // [DV]
    float* us = vs + DV;                    // [DV]
    float* part = us + DV;                  // [NG][DV]
    const int c4n = DV >> 2, NG = 256 / c4n;
    float* qs = part + (size_t)NG * DV;     // [D4]
    float* ks = qs + D4;
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int t = cu_q[seq], C = 2 * G * D + H * DV, r = H / G, grp = h / r;
    float* st = state + ((size_t)slots[seq] * H + h) * D * DV;
    const int g = tid / c4n, col = (tid - g * c4n) << 2;
    const bool owner = g < NG;
    const float* row = proj + (size_t)t * ld;
    const int pos = positions[t];
    float* slot = ring + (size_t)ring_slots[seq] * K * C;
    auto channel = [&](int i) { return i < D ? grp * D + i : i < 2 * D ? G * D + grp * D + i - D : 2 * G * D + h * DV + i - 2 * D; };
    const float b_in = row[C + H * DV + h], a_in = row[C + H * DV + H + h], rate_h = rate[h], shift_h = shift[h];
    float x[2], tap[2][4], kept[2][3];
    if constexpr (FEW) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int i = tid + 256 * n, c = channel(i);
            const bool in = i < 2 * D + DV;
            x[n] = in ? row[c] : 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) tap[n][j] = in && j < K ? wt[(size_t)(K - 1 - j) * C + c] : 0.f;
#pragma unroll
            for (int j = 1; j < 4; ++j) kept[n][j - 1] = in && j < K && j <= pos ? slot[(size_t)((pos - j) % K) * C + c] : 0.f;
        }
    }
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + i * NG;
        S[i] = owner && d < D ? *reinterpret_cast<const float4*>(st + (size_t)d * DV + col) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float z0 = tid < DV ? row[C + h * DV + tid] : 0.f, w0 = tid < DV ? weight[(size_t)h * DV + tid] : 0.f;
    auto take = [&](int i, int c, float in, float y) {
        // the heads of a group share their q and k channels: one of them keeps the input (in the row that nobody reads now)
        if (K > 1 && (i >= 2 * D || h == grp * r)) slot[(size_t)(pos % K) * C + c] = in;
        (i < D ? qs[i] : i < 2 * D ? ks[i - D] : vs[i - 2 * D]) = gd_silu(y);
    };
    if constexpr (FEW) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int i = tid + 256 * n;
            float y = tap[n][0] * x[n];
#pragma unroll
            for (int j = 1; j < 4; ++j) y = fmaf(tap[n][j], kept[n][j - 1], y);
            if (i < 2 * D + DV) take(i, channel(i), x[n], y);
        }
    } else {
        for (int i = tid; i < 2 * D + DV; i += 256) {
            const int c = channel(i);
            const float in = row[c];
            float y = wt[(size_t)(K - 1) * C + c] * in;
            for (int j = 1; j < K && j <= pos; ++j) y = fmaf(wt[(size_t)(K - 1 - j) * C + c], slot[(size_t)((pos - j) % K) * C + c], y);
            take(i, c, in, y);
        }
    }
    const float beta = gd_sigmoid(b_in), dec = gd_decay(a_in, rate_h, shift_h);
    __syncthreads();
    float qq = 0.f, kk = 0.f;               // (every warp for itself)
    for (int e = lane; e < D; e += 32) {
        qq = fmaf(qs[e], qs[e], qq);
        kk = fmaf(ks[e], ks[e], kk);
    }
    const float inv_q = 1.f / (sqrtf(warp_sum(qq) + GD_UNIT_EPS) * sqrtf((float)D)), inv_k = 1.f / sqrtf(warp_sum(kk) + GD_UNIT_EPS);
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
    if (owner) *reinterpret_cast<float4*>(part + (size_t)g * DV + col) = acc;
    __syncthreads();
    for (int c = tid; c < DV; c += 256) {
        float p = 0.f;
        for (int i = 0; i < NG; ++i) p += part[(size_t)i * DV + c];
        us[c] = beta * (vs[c] - dec * inv_k * p) * inv_k;      // (times the key's length: the update takes ks as it lies)
    }
    __syncthreads();
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner) {
        const float4 u = *reinterpret_cast<const float4*>(us + col);
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int d = g + i * NG;
            if (d < D) {
                const float kd = ks[d], qd = qs[d];
                S[i].x = fmaf(dec, S[i].x, kd * u.x); S[i].y = fmaf(dec, S[i].y, kd * u.y);
                S[i].z = fmaf(dec, S[i].z, kd * u.z); S[i].w = fmaf(dec, S[i].w, kd * u.w);
                *reinterpret_cast<float4*>(st + (size_t)d * DV + col) = S[i];
                acc.x = fmaf(qd, S[i].x, acc.x); acc.y = fmaf(qd, S[i].y, acc.y);
                acc.z = fmaf(qd, S[i].z, acc.z); acc.w = fmaf(qd, S[i].w, acc.w);
            }
        }
        *reinterpret_cast<float4*>(part + (size_t)g * DV + col) = acc;
    }
    __syncthreads();
    float sq = 0.f;
    for (int c = tid; c < DV; c += 256) {
        float o = 0.f;
        for (int i = 0; i < NG; ++i) o += part[(size_t)i * DV + c];
        o *= inv_q;
        us[c] = o;                          // (read again by this thread alone)
        sq = fmaf(o, o, sq);
    }
    const float inv_rms = 1.f / sqrtf(block_sum(sq, red) / (float)DV + eps);
    for (int c = tid; c < DV; c += 256)
        out[(size_t)t * ldo + (size_t)h * DV + c] =
            from_f32<T>(us[c] * inv_rms * (c == tid ? w0 : weight[(size_t)h * DV + c]) * gd_silu(c == tid ? z0 : row[C + h * DV + c]));
}

static size_t gated_delta_step_smem(int D, int DV) {
    const int NG = 256 / (DV / 4);
    return ((size_t)(2 + NG) * DV + 2 * ((D + 3) & ~3)) * sizeof(float);
}

// 1 if acv_gated_delta_step runs these sizes
ACV_API int acv_gated_delta_step_takes(int D, int DV) {
    if (DV < 4 || DV % 4 || DV > 1024 || D < 1 || gated_delta_step_smem(D, DV) > 48 * 1024) return 0;
    const int NG = 256 / (DV / 4);
    return (D + NG - 1) / NG <= 32;
}

// out: rows of H*DV elements at ldo (float or bfloat16): each head's o / sqrt(mean(o^2) + eps), times weight (float [H*DV]),
// times silu(z).  state: float [slots][H][D][DV]; the rest as acv_gated_delta_blocks takes it; every request brings one token.
ACV_API int acv_gated_delta_step(const float* proj, int ld, const float* wt, const float* rate, const float* shift,
                                 const float* weight, float eps, float* ring, const int* ring_slots, float* state,
                                 const int* slots, const int* positions, const int* cu_q, void* out, int ldo, int n_seqs, int G,
                                 int H, int D, int DV, int K, int dtype, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (G <= 0 || H <= 0 || H > 65535 || H % G || K < 1 || !acv_gated_delta_step_takes(D, DV) || ld < 2 * G * D + 2 * H * DV + 2 * H)
        return ACV_ERR_SIZE;
    if ((uintptr_t)state & 15) return ACV_ERR_ALIGN;
    const int NG = 256 / (DV / 4), rows = (D + NG - 1) / NG;
    const size_t smem = gated_delta_step_smem(D, DV);
    const dim3 grid(n_seqs, H);
    const bool few = K <= 4 && 2 * D + DV <= 512;
#define GS_LAUNCH(TT, N, F)                                                                                                 \
    acv_launch(PDL_ATTN, gated_delta_step_kernel<TT, N, F>, grid, 256, smem, stream, proj, ld, wt, rate, shift, weight, eps, \
               ring, ring_slots, state, slots, positions, cu_q, (TT*)out, ldo, G, H, D, DV, K)
#define GS_CASE(N)                                                                                                          \
    if (rows <= N) {                                                                                                        \
        if (dtype == ACV_F32) {                                                                                             \
            if (few) GS_LAUNCH(float, N, true); else GS_LAUNCH(float, N, false);                                            \
        } else if (dtype == ACV_BF16) {                                                                                     \
            if (few) GS_LAUNCH(bf16, N, true); else GS_LAUNCH(bf16, N, false);                                              \
        } else {                                                                                                            \
            return ACV_ERR_DTYPE;                                                                                           \
        }                                                                                                                   \
        return acv_launch_status();                                                                                         \
    }
    GS_CASE(1) GS_CASE(2) GS_CASE(4) GS_CASE(8) GS_CASE(16) GS_CASE(32)
#undef GS_CASE
#undef GS_LAUNCH
    return ACV_ERR_SIZE;
}
