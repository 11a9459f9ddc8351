// One-token requests over kept latent rows (see latent_attention_tc.cu, whose arguments and merge they share).
//
// A CTA is one request (or a share of its rows) with up to 16 heads: the 16 rows of mma.sync m16n8k16.  Eight warps; the
// queries' fragments stay in registers for the whole walk (NK steps of 16 elements), key tiles of 64 rows come by bulk
// copies, two tiles ahead.  For a tile each warp makes the scores of eight keys (four chains of products), the warps
// exchange their row maxima and weights through shared memory, and each multiplies all 64 weights with its own
// NDV * 16 value columns.
#pragma once

#define LD_BN 64
#define LD_NB 3
#define LD_THREADS 256

template <int NK, int NDV>
__global__ void __launch_bounds__(LD_THREADS, 1)
attn_latent_dec_kernel(const LatentArgs a) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ __align__(8) uint64_t full_s[LD_NB];
    __shared__ int abort_s;
    const int ROW = a.ROW, KR = a.KR;
    const int DP = (ROW + 15) & ~15, KRP = (KR + 15) & ~15, nk = DP >> 4;
    const int QP = DP * 2 + 16;                 // bytes of a padded row
    constexpr int PP = (LD_BN + 8) * 2;
    unsigned char* k_s = smem;                                      // [LD_NB][LD_BN][QP]
    unsigned char* p_s = k_s + (size_t)LD_NB * LD_BN * QP;          // [16][PP]
    float* mx_s = reinterpret_cast<float*>(p_s + 16 * PP);          // [16][8]
    float* l_s = mx_s + 16 * 8;                                     // [16][8]

    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int hb = blockIdx.x % a.HB, u = blockIdx.x / a.HB;
    const int i = u / a.n_split, split = u % a.n_split;
    const int part = a.n_split > 1 ? u : -1;    // >= 0: this CTA leaves a partial result at that index
    const int seq = a.dec_seqs[i], tok = a.dec_tokens[i], pos = a.kv_len[seq] - 1;
    const int h_first = hb * 16, nh = min(16, a.NH - h_first);
    if (pos < 0) {                              // a padded slot of a captured batch: nothing is kept for it
        if (part >= 0) {
            if (tid < nh) {
                a.part_ml[((size_t)part * a.NH + h_first + tid) * 2] = -INFINITY;
                a.part_ml[((size_t)part * a.NH + h_first + tid) * 2 + 1] = 0.f;
            }
            return;
        }
        for (int e = tid; e < nh * KR; e += LD_THREADS)
            a.out[(size_t)tok * a.out_stride + (size_t)h_first * KR + e] = from_f32<bf16>(0.f);
        return;
    }
    const int* bt = a.block_table + (size_t)(a.bt_rows ? a.bt_rows[seq] : seq) * a.bt_stride;
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int j_first = lo & ~(LD_BN - 1);
    const int n_all = (pos - j_first) / LD_BN + 1;
    const int per_split = (n_all + a.n_split - 1) / a.n_split;
    const int t_first = split * per_split, n_t = min(n_all, t_first + per_split);

    const uint32_t full0 = gt_smem(full_s);
    if (DP > ROW)                               // a row's last 16 bytes, which no copy brings
        for (int r = tid; r < LD_NB * LD_BN; r += LD_THREADS) *reinterpret_cast<uint4*>(k_s + (size_t)r * QP + ROW * 2) = make_uint4(0, 0, 0, 0);
    // the queries wait in the last buffer until their fragments are read
    unsigned char* q_s = k_s + (size_t)(LD_NB - 1) * LD_BN * QP;
    const int CH = DP / 8;
    for (int id = tid; id < 16 * CH; id += LD_THREADS) {
        const int c = id % CH, R = id / CH;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (R < nh && c * 8 < ROW)
            v = *reinterpret_cast<const uint4*>(a.q + (size_t)tok * a.q_stride + (size_t)(h_first + R) * ROW + c * 8);
        *reinterpret_cast<uint4*>(q_s + (size_t)R * QP + c * 16) = v;
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");        // (copies follow where these writes are)
    if (tid == 0) {
        abort_s = 0;
        for (int b = 0; b < LD_NB; ++b) mbar_init(full0 + 8 * b, LD_BN);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    // a thread a row: a bulk copy counted at the buffer's barrier, or zeros where no query sees the row (or it has no page)
    auto load_keys = [&](int t) {
        if (tid >= LD_BN) return;
        const int j = j_first + t * LD_BN + tid, buf = (t - t_first) % LD_NB;
        unsigned char* dst = k_s + ((size_t)buf * LD_BN + tid) * QP;
        const uint32_t bar = full0 + 8 * buf;
        int pg = -1;
        if (j <= pos && j >= lo) pg = bt[j / a.page_size];
        if (pg >= 0 && pg < a.num_pages) {
            const bf16* src = a.pages + ((size_t)pg * a.page_size + (j % a.page_size)) * ROW;
            mbar_expect_tx(bar, ROW * 2);       // (arrives)
            asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                         ::"r"(smem_u32(dst)), "l"(src), "r"(ROW * 2), "r"(bar) : "memory");
        } else {
            for (int c = 0; c < ROW / 8; ++c) *reinterpret_cast<uint4*>(dst + c * 16) = make_uint4(0, 0, 0, 0);
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(bar);
        }
    };
    for (int t = t_first; t < n_t && t < t_first + LD_NB - 1; ++t) load_keys(t);

    const int mi = lane >> 3, lr = lane & 7;
    const int r_lo = lane >> 2, c_lo = (lane & 3) * 2;
    uint32_t qf[NK][4];
#pragma unroll
    for (int kd = 0; kd < NK; ++kd) {
        if (kd < nk) ldmatrix_x4(qf[kd], smem_u32(q_s) + ((mi & 1) * 8 + lr) * QP + (kd * 2 + (mi >> 1)) * 16);
        else qf[kd][0] = qf[kd][1] = qf[kd][2] = qf[kd][3] = 0u;
    }
    const float sc_log2 = a.scale * LT_LOG2E;
    const uint32_t pb = smem_u32(p_s);
    float acc[2 * NDV][4];
#pragma unroll
    for (int c = 0; c < 2 * NDV; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[c][e] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

    for (int t = t_first; t < n_t; ++t) {
        const int turn = t - t_first, buf = turn % LD_NB;
        const bool there = mbar_wait(full0 + 8 * buf, (turn / LD_NB) & 1, &abort_s);
        if (!__syncthreads_and(there)) {        // (also: everyone is done with the tile before, and has read its queries)
            if (tid == 0) atomicExch(a.status, LT_STATUS);
            for (int w = t; w < n_t && w < t + LD_NB - 1; ++w)      // the copies that are under way end before the block does
                mbar_wait(full0 + 8 * ((w - t_first) % LD_NB), ((w - t_first) / LD_NB) & 1, &abort_s);
            return;
        }
        if (t + LD_NB - 1 < n_t) load_keys(t + LD_NB - 1);
        const uint32_t kb = smem_u32(k_s + (size_t)buf * LD_BN * QP);
        // scores of keys warp*8 .. +7: four chains
        float s4[4][4];
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) s4[c][e] = 0.f;
        const uint32_t krow = kb + (warp * 8 + lr) * QP + mi * 16;
#pragma unroll
        for (int k2 = 0; k2 < NK / 2; ++k2) {
            if (2 * k2 < nk) {
                uint32_t b[4];                  // eight keys, two steps of 16 elements
                ldmatrix_x4(b, krow + k2 * 64);
                mma_bf16(s4[(2 * k2) & 3], qf[2 * k2], b[0], b[1]);
                if (2 * k2 + 1 < nk) mma_bf16(s4[(2 * k2 + 1) & 3], qf[2 * k2 + 1], b[2], b[3]);
            }
        }
        const int key = warp * 8 + c_lo, j = j_first + t * LD_BN + key;
        float s[4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const bool seen = j + (e & 1) <= pos && j + (e & 1) >= lo;
            s[e] = seen ? ((s4[0][e] + s4[1][e]) + (s4[2][e] + s4[3][e])) * sc_log2 : -INFINITY;
            mx[e >> 1] = fmaxf(mx[e >> 1], s[e]);
        }
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
            mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
            mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
            if ((lane & 3) == 0) mx_s[(r_lo + hh * 8) * 8 + warp] = mx[hh];
        }
        __syncthreads();
        float alpha[2], m_use[2];
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
            const float4 x = reinterpret_cast<const float4*>(mx_s + (r_lo + hh * 8) * 8)[0], y = reinterpret_cast<const float4*>(mx_s + (r_lo + hh * 8) * 8)[1];
            const float m_new = fmaxf(m_run[hh], fmaxf(fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w)), fmaxf(fmaxf(y.x, y.y), fmaxf(y.z, y.w))));
            m_use[hh] = m_new == -INFINITY ? 0.f : m_new;
            alpha[hh] = fast_exp2(m_run[hh] - m_use[hh]);
            m_run[hh] = m_new;
            const float p0 = fast_exp2(s[2 * hh] - m_use[hh]), p1 = fast_exp2(s[2 * hh + 1] - m_use[hh]);
            l_run[hh] = l_run[hh] * alpha[hh] + (p0 + p1);
            *reinterpret_cast<uint32_t*>(p_s + (size_t)(r_lo + hh * 8) * PP + key * 2) = pack_bf16(p0, p1);
        }
        if (alpha[0] != 1.f || alpha[1] != 1.f) {
#pragma unroll
            for (int c = 0; c < 2 * NDV; ++c) {
                acc[c][0] *= alpha[0]; acc[c][1] *= alpha[0];
                acc[c][2] *= alpha[1]; acc[c][3] *= alpha[1];
            }
        }
        __syncthreads();
#pragma unroll
        for (int kp = 0; kp < LD_BN / 16; ++kp) {
            uint32_t pa[4];
            ldmatrix_x4(pa, pb + ((mi & 1) * 8 + lr) * PP + (kp * 2 + (mi >> 1)) * 16);
#pragma unroll
            for (int nd = 0; nd < NDV; ++nd) {
                const int c16 = warp * NDV + nd;
                if (c16 * 16 < KRP) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, kb + (kp * 16 + (mi & 1) * 8 + lr) * QP + (c16 * 2 + (mi >> 1)) * 16);
                    mma_bf16(acc[2 * nd], pa, b[0], b[1]);
                    mma_bf16(acc[2 * nd + 1], pa, b[2], b[3]);
                }
            }
        }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
        l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
        if ((lane & 3) == 0) l_s[(r_lo + hh * 8) * 8 + warp] = l_run[hh];
    }
    __syncthreads();
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        const int R = r_lo + hh * 8;
        if (R >= nh) continue;
        float l = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) l += l_s[R * 8 + w];
        const int col = warp * NDV * 16 + c_lo;
        if (part >= 0) {        // unnormalised sums, running maximum and sum, for the merge
            const size_t at = (size_t)part * a.NH + h_first + R;
#pragma unroll
            for (int c = 0; c < 2 * NDV; ++c)
                if (col + c * 8 < KR) *reinterpret_cast<float2*>(a.part_acc + at * KR + col + c * 8) = make_float2(acc[c][2 * hh], acc[c][2 * hh + 1]);
            if (warp == 0 && (lane & 3) == 0) {
                a.part_ml[at * 2] = m_run[hh];
                a.part_ml[at * 2 + 1] = l;
            }
            continue;
        }
        float inv = l > 0.f ? 1.f / l : 0.f;
        if (a.sinks) {
            const float sk = a.sinks[h_first + R] * LT_LOG2E, M = fmaxf(m_run[hh], sk);
            const float al = fast_exp2(m_run[hh] - M);
            inv = al / fmaf(l, al, fast_exp2(sk - M));
        }
        bf16* o = a.out + (size_t)tok * a.out_stride + (size_t)(h_first + R) * KR + col;
#pragma unroll
        for (int c = 0; c < 2 * NDV; ++c)
            if (col + c * 8 < KR)
                *reinterpret_cast<__nv_bfloat162*>(o + c * 8) = __floats2bfloat162_rn(acc[c][2 * hh] * inv, acc[c][2 * hh + 1] * inv);
    }
}

static size_t latent_dec_smem(int ROW) {
    const size_t QP = ((ROW + 15) & ~15) * 2 + 16;
    return (size_t)LD_NB * LD_BN * QP + 16 * (LD_BN + 8) * 2 + 2 * 16 * 8 * sizeof(float);
}
static bool latent_dec_takes(int ROW, int KR) { return ROW % 8 == 0 && KR % 8 == 0 && KR <= ROW && KR <= 512 && ROW <= 576; }

// a.HB, a.n_dec, a.n_split and the rest of the arguments are set; the merge follows by the caller
template <int NK, int NDV>
static int launch_latent_dec(const LatentArgs& a, cudaStream_t stream) {
    static AcvSmemConfig cfg;
    const size_t smem = latent_dec_smem(a.ROW);
    if (int rc = acv_ensure_smem(cfg, attn_latent_dec_kernel<NK, NDV>, (int)smem)) return rc;
    acv_launch(PDL_ATTN, attn_latent_dec_kernel<NK, NDV>, dim3(a.n_dec * a.n_split * a.HB), dim3(LD_THREADS), smem, stream, a);
    return 0;
}
