// Attention whose keys and values are made from one kept latent per token.
//
// Per token the layer keeps one row [c | r]: c = the normed latent (KR elements), r = a rotated key part (R elements)
// that all heads share.  Head h's key is [W_uk,h c | r] and its value W_uv,h c.  The products with W_uk and W_uv move
// to the query's side, where they cost one product per query instead of one per (query, key):
//
//   <q_h, W_uk,h c> = <W_uk,h^T q_h, c>             the query the kept rows are scored with: [W_uk,h^T q_h | q_rot,h]
//   sum_j p_j W_uv,h c_j = W_uv,h (sum_j p_j c_j)   the weighted sum is taken over the latents, then projected
//
// so the attention itself is one key/value head of KR + R elements whose values are the first KR elements of the same
// rows (the generic paged kernel with v_pages == k_pages), read by every query head.
//
// acv_latent_prepare, one block a token:
//   kv row [KR + R] of the down projection: c = kv[:KR] / sqrt(mean(kv[:KR]^2) + eps) * w (32-bit), r = rot(kv[KR:]);
//     [c | r] goes into the token's row of its page (a page index < 0 writes nothing);
//   q rows [H][D + R]: rot(q_h[D:]) goes to q_out[h][KR:], beside the place where the caller's per-head product leaves
//     W_uk,h^T q_h[:D].
// rot turns the interleaved pairs (2i, 2i+1), 2i < rot, or with `halves` the pairs (i, i + rot/2), by the angle of pair i at
// the token's position (cos and sin from a float table [positions][rot]: rot/2 cosines, then rot/2 sines); elements from
// rot on pass unchanged.  A layer that reads rows kept by another one gives no kv: queries only.
#include "common.cuh"

template <typename T>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const T* __restrict__ q, int q_stride, T* __restrict__ q_out, int qo_stride,
                      const T* __restrict__ kv, int kv_stride, const float* __restrict__ w, float eps,
                      const float* __restrict__ cos_sin, int rot, int table_rows, const int* __restrict__ positions,
                      const int* __restrict__ seq_of_token, const int* __restrict__ block_table, int bt_stride,
                      const int* __restrict__ bt_rows, T* __restrict__ pages, int page_size, int num_pages, int H, int D, int R,
                      int KR, int halves, int full, int vec) {
    extern __shared__ float row[];          // [KR] the latent part of the kv row
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, nthr = blockDim.x;
    const int warp = tid >> 5, lane = tid & 31, nw = nthr >> 5, half = rot >> 1;
    const int at = positions[t], pos = min(at, table_rows - 1);
    const float* cs = cos_sin + (size_t)pos * rot;
    float c0 = 1.f, s0 = 0.f;               // the lane's first pair
    if (lane < half) { c0 = cs[lane]; s0 = cs[half + lane]; }
    int pg = -1;
    if (pages && kv) {
        const int seq = seq_of_token[t];
        pg = block_table[(size_t)(bt_rows ? bt_rows[seq] : seq) * bt_stride + at / page_size];
    }
    // R elements turned, by a warp: a lane a pair
    auto turn = [&](const T* src, T* dst) {
        for (int i = lane; i < half; i += 32) {
            const float c = i == lane ? c0 : cs[i], s = i == lane ? s0 : cs[half + i];
            const int a = halves ? i : 2 * i, b = halves ? i + half : 2 * i + 1;
            const float u = to_f32(src[a]), v = to_f32(src[b]);
            dst[a] = from_f32<T>(fmaf(u, c, -v * s));
            dst[b] = from_f32<T>(fmaf(v, c, u * s));
        }
        for (int e = rot + lane; e < R; e += 32) dst[e] = src[e];
    };
    const T* kvr = kv + (size_t)t * kv_stride;
    float ss = 0.f;
    if (kv)
        for (int e = tid; e < KR; e += nthr) {
            const float v = to_f32(kvr[e]);
            row[e] = v;
            ss = fmaf(v, v, ss);
        }
    for (int h = warp; h < H; h += nw) {
        const T* src = q + (size_t)t * q_stride + (size_t)h * (D + R);
        if (full) {             // whole heads [plain | rotated | zeros] of `full` elements
            T* dst = q_out + (size_t)t * qo_stride + (size_t)h * full;
            constexpr int P = 8 / (int)sizeof(T);
            if (vec) {          // plain parts in 8-byte pieces
                for (int e = lane * P; e < D; e += 32 * P) *reinterpret_cast<uint2*>(dst + e) = *reinterpret_cast<const uint2*>(src + e);
            } else {
                for (int e = lane; e < D; e += 32) dst[e] = src[e];
            }
            turn(src + D, dst + D);
            for (int e = D + R + lane; e < full; e += 32) dst[e] = from_f32<T>(0.f);
        } else {
            turn(src + D, q_out + (size_t)t * qo_stride + (size_t)h * (KR + R) + KR);
        }
    }
    if (!kv) return;
    ss = block_sum(ss, red);                // (meets the block: row is whole)
    if (pg < 0 || pg >= num_pages) return;
    const float inv = 1.f / sqrtf(ss / (float)KR + eps);
    T* dst = pages + ((size_t)pg * page_size + at % page_size) * (KR + R);
    for (int e = tid; e < KR; e += nthr) dst[e] = from_f32<T>(row[e] * inv * w[e]);
    if (warp == nw - 1) turn(kvr + KR, dst + KR);
}

// q: rows of H*(D+R) at q_stride; q_out: rows of H*(KR+R) at qo_stride; kv: rows of KR+R at kv_stride; w float [KR];
// cos_sin float [table_rows][rot]; pages [num_pages][1][page_size][KR+R] (null: nothing is kept, queries only).
// full > 0: q_out is rows of H heads of `full` elements, [plain | rotated | zeros] (queries for keys that are written out).
ACV_API int acv_latent_prepare(const void* q, int q_stride, void* q_out, int qo_stride, const void* kv, int kv_stride,
                               const float* w, float eps, const float* cos_sin, int rot, int table_rows,
                               const int* positions, const int* seq_of_token, const int* block_table, int bt_stride,
                               const int* bt_rows, void* pages, int page_size, int num_pages, int T_tokens, int H, int D,
                               int R, int KR, int dtype, int halves, int full, cudaStream_t stream) {
    if (T_tokens <= 0) return 0;
    if (H <= 0 || D < 0 || R <= 0 || KR <= 0 || rot < 0 || rot > R || (rot & 1) || (full && full < D + R) || (rot && (!cos_sin || table_rows <= 0)))
        return ACV_ERR_SIZE;
    const size_t smem = (size_t)KR * sizeof(float);
    if (smem > 200 * 1024) return ACV_ERR_SIZE;
    const int threads = 256;
    const int piece = dtype == ACV_F32 ? 2 : 4;         // elements of 8 bytes
    const int vec = D % piece == 0 && R % piece == 0 && full % piece == 0 && q_stride % piece == 0 && qo_stride % piece == 0 &&
                    !(((uintptr_t)q | (uintptr_t)q_out) & 7);
#define LP_LAUNCH(T)                                                                                                    \
    do {                                                                                                                \
        if (smem > 48 * 1024) {                                                                                         \
            static AcvSmemConfig cfg;                                                                                   \
            const int e = acv_ensure_smem(cfg, latent_prepare_kernel<T>, (int)smem);                                    \
            if (e) return e;                                                                                            \
        }                                                                                                               \
        acv_launch(PDL_ROPE, latent_prepare_kernel<T>, T_tokens, threads, smem, stream, (const T*)q, q_stride, (T*)q_out, \
                   qo_stride, (const T*)kv, kv_stride, w, eps, cos_sin, rot, table_rows, positions, seq_of_token,       \
                   block_table, bt_stride, bt_rows, (T*)pages, page_size, num_pages, H, D, R, KR, halves, full, vec);                      \
    } while (0)
    if (dtype == ACV_F32) LP_LAUNCH(float);
    else if (dtype == ACV_BF16) LP_LAUNCH(bf16);
    else return ACV_ERR_DTYPE;
#undef LP_LAUNCH
    return acv_launch_status();
}

// ----------------------------------------------------------------------------- RMS norm of rows at any stride
// out[r][:] = x[r][:] / sqrt(mean(x[r]^2) + eps) * w, 32-bit, rounded once; x and out are column ranges of wider
// matrices (a latent inside a stacked projection's output).  One block a row.
template <typename T>
__global__ void rmsnorm_rows_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ w, float eps,
                                    T* __restrict__ out, int ldo, int H) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const T* xr = x + (size_t)blockIdx.x * ldx;
    T* o = out + (size_t)blockIdx.x * ldo;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_f32(xr[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = from_f32<T>(to_f32(xr[i]) * inv * (w ? w[i] : 1.f));
}

ACV_API int acv_rmsnorm_rows(const void* x, int ldx, const float* w, float eps, void* out, int ldo, int n_rows, int H,
                             int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (H <= 0) return ACV_ERR_SIZE;
    const int threads = H >= 2048 ? 256 : 128;
    if (dtype == ACV_F32)
        acv_launch(PDL_NORM, rmsnorm_rows_kernel<float>, n_rows, threads, 0, stream, (const float*)x, ldx, w, eps, (float*)out, ldo, H);
    else if (dtype == ACV_BF16)
        acv_launch(PDL_NORM, rmsnorm_rows_kernel<bf16>, n_rows, threads, 0, stream, (const bf16*)x, ldx, w, eps, (bf16*)out, ldo, H);
    else
        return ACV_ERR_DTYPE;
    return acv_launch_status();
}
