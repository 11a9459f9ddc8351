// One-token requests over kept latent rows (see latent_attention_tc.cu, whose arguments and merge they share).
//
// A CTA is one request (or a share of its rows) with up to 16 heads: the 16 rows of mma.sync m16n8k16.  Eight warps; the
// queries' fragments stay in registers for the whole walk (NK steps of 16 elements), key tiles of 64 rows come by TMA, two
// tiles ahead: a box is 64 elements (one 128-byte swizzle row) of a page's rows, or of 64 of them.  For a tile each warp makes the scores of eight keys (four chains of products), the warps
// exchange their row maxima and weights through shared memory, and each multiplies all 64 weights with its own
// NDV * 16 value columns.
#pragma once

#define LD_BN 64
#define LD_NB 3
#define LD_THREADS 256
#define LD_ATOM (LD_BN * 128)    // bytes of 64 elements of a tile's rows

// EXACT: rows of NK * 16 elements with latents of NDV * 128 (sizes known when compiled); otherwise up to that
template <int NK, int NDV, bool EXACT>
__global__ void __launch_bounds__(LD_THREADS, 1)
attn_latent_dec_kernel(const __grid_constant__ CUtensorMap rows, const LatentArgs a) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = smem_raw + ((1024u - (gt_smem(smem_raw) & 1023u)) & 1023u);
    __shared__ __align__(8) uint64_t full_s[LD_NB];
    __shared__ int abort_s;
    const int ROW = EXACT ? NK * 16 : a.ROW, KR = EXACT ? NDV * 128 : a.KR;
    const int DP = (ROW + 15) & ~15, KRP = (KR + 15) & ~15, nk = DP >> 4;
    const int NA = (ROW + 63) >> 6;             // 64-element pieces of a row
    constexpr int PP = (LD_BN + 8) * 2;
    unsigned char* k_s = smem;                                      // [LD_NB][NA][LD_BN][128 bytes, swizzled]
    unsigned char* p_s = k_s + (size_t)LD_NB * NA * LD_ATOM;        // [16][PP]
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
    // the queries wait in the last buffer until their fragments are read
    const int QP = DP * 2 + 16;
    unsigned char* q_s = k_s + (size_t)(LD_NB - 1) * NA * LD_ATOM;
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
        for (int b = 0; b < LD_NB; ++b) mbar_init(full0 + 8 * b, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    // Warp 0 loads: a lane a page of the tile (or 64 rows of one), looked up a tile earlier.  A page that is not there is a
    // place outside the pool, which reads as zeros; rows behind the last token of a page hold older, finite numbers.
    const int box = min(a.page_size, LD_BN), n_box = LD_BN / box;
    auto row_of = [&](int t) {                  // the box's first row in the pool
        const int j = j_first + t * LD_BN + lane * box;
        if (warp || lane >= n_box || t >= n_t || j > pos || j + box <= lo) return -LD_BN;
        const int pg = bt[j / a.page_size];
        return pg >= 0 && pg < a.num_pages ? pg * a.page_size + j % a.page_size : -LD_BN;
    };
    int row = row_of(t_first);
    auto load_keys = [&](int t) {
        if (warp) return;
        const int buf = (t - t_first) % LD_NB, next = row_of(t + 1);
        const uint32_t dst = smem_u32(k_s) + buf * NA * LD_ATOM, bar = full0 + 8 * buf;
        if (lane == 0) mbar_expect_tx(bar, NA * LD_ATOM);
        __syncwarp();
        if (lane < n_box)
            for (int c = 0; c < NA; ++c) tma_load_2d(dst + c * LD_ATOM + lane * box * 128, &rows, bar, c * 64, row);
        row = next;
    };
    for (int t = t_first; t < n_t && t < t_first + LD_NB - 1; ++t) load_keys(t);

    const int mi = lane >> 3, lr = lane & 7;
    const int r_lo = lane >> 2, c_lo = (lane & 3) * 2;
    uint32_t qf[NK][4];
#pragma unroll
    for (int kd = 0; kd < NK; ++kd) {
        if (EXACT || kd < nk) ldmatrix_x4(qf[kd], smem_u32(q_s) + ((mi & 1) * 8 + lr) * QP + (kd * 2 + (mi >> 1)) * 16);
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
        const uint32_t kb = smem_u32(k_s) + buf * NA * LD_ATOM;
        // scores of keys warp*8 .. +7: four chains
        float s4[4][4];
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) s4[c][e] = 0.f;
        const uint32_t krow = kb + (warp * 8 + lr) * 128, kx[2] = {(uint32_t)(mi ^ lr) << 4, (uint32_t)((4 + mi) ^ lr) << 4};
#pragma unroll
        for (int k2 = 0; k2 < NK / 2; ++k2) {
            if (EXACT || 2 * k2 < nk) {
                uint32_t b[4];                  // eight keys, two steps of 16 elements
                ldmatrix_x4(b, krow + (k2 >> 1) * LD_ATOM + kx[k2 & 1]);
                mma_bf16(s4[(2 * k2) & 3], qf[2 * k2], b[0], b[1]);
                if (EXACT || 2 * k2 + 1 < nk) mma_bf16(s4[(2 * k2 + 1) & 3], qf[2 * k2 + 1], b[2], b[3]);
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
                if (EXACT || c16 * 16 < KRP) {
                    uint32_t b[4];
                    const int ch = c16 * 2 + (mi >> 1);
                    ldmatrix_x4_trans(b, kb + (ch >> 3) * LD_ATOM + (kp * 16 + (mi & 1) * 8 + lr) * 128 + (((ch & 7) ^ lr) << 4));
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
    return (size_t)LD_NB * ((ROW + 63) / 64) * LD_ATOM + 16 * (LD_BN + 8) * 2 + 2 * 16 * 8 * sizeof(float) + 1024;
}
static bool latent_dec_takes(int ROW, int KR, int page_size, int num_pages) {
    return ROW % 8 == 0 && KR % 8 == 0 && KR <= ROW && KR <= 512 && ROW <= 576 && page_size >= 8 && page_size <= 1024 &&
           !(page_size & (page_size - 1)) && (long long)num_pages * page_size <= 0x7fffffffLL;
}

// a.HB, a.n_dec, a.n_split and the rest of the arguments are set; the merge follows by the caller
template <int NK, int NDV, bool EXACT>
static int launch_latent_dec(const LatentArgs& a, cudaStream_t stream) {
    static AcvSmemConfig cfg;
    const size_t smem = latent_dec_smem(a.ROW);
    if (int rc = acv_ensure_smem(cfg, attn_latent_dec_kernel<NK, NDV, EXACT>, (int)smem)) return rc;
    CUtensorMap rows;
    if (int rc = make_map(&rows, a.pages, a.num_pages * a.page_size, a.ROW, a.ROW, a.page_size < LD_BN ? a.page_size : LD_BN)) return rc;
    acv_launch(PDL_ATTN, attn_latent_dec_kernel<NK, NDV, EXACT>, dim3(a.n_dec * a.n_split * a.HB), dim3(LD_THREADS), smem, stream, rows, a);
    return 0;
}
