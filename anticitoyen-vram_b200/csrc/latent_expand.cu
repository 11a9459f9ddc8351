// Latent attention for portions of prompts with keys and values written out.
//
// Over kept rows [c | r] (latent_attention.cu) every score costs KR + R multiply-adds and every weighted sum KR, for every
// head: right for a token that reads a long context once, wasteful when many tokens read the same context.  For a
// portion the keys [W_uk,h c | r] and values W_uv,h c of the request's context are made once (one product over its kept
// rows) and laid out as pages of 128 tokens with a key/value head for each query head, which the tensor-core attention for
// portions (attention_tc.cu) reads.  Keys and values are padded with zeros to its head size HD.
//
//   acv_latent_context   the kept rows of the portions' requests, out of the cache's pages, 128 rows a page, zeros behind a
//                        request's last token
//   acv_latent_pack      the product's rows [K (H D) | V (H DV)] and the rotated parts to pages [page][H][128][HD]
//   acv_latent_pick      one-token requests beside portions: their queries' plain parts, and their rotated parts into the
//                        queries that meet the kept rows
//   acv_heads_gated      heads [rows][H][HD] to columns of wider rows, times sigmoid of a gate (or not), to listed rows (or all)
#include "common.cuh"

#define LX_PAGE 128

// grid (pages of context, 128 / 8): a warp a row.  ROW elements a row; 16-byte pieces where `vec`.
__global__ void __launch_bounds__(256)
latent_context_kernel(const bf16* __restrict__ pages, const int* __restrict__ page_seq, const int* __restrict__ page_idx,
                      const int* __restrict__ kv_len, const int* __restrict__ block_table, int bt_stride,
                      const int* __restrict__ bt_rows, bf16* __restrict__ out, int ROW, int page_size, int num_pages, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seq = page_seq[blockIdx.x], r = blockIdx.y * 8 + warp, j = page_idx[blockIdx.x] * LX_PAGE + r;
    bf16* dst = out + ((size_t)blockIdx.x * LX_PAGE + r) * ROW;
    int pg = -1;
    if (j < kv_len[seq]) pg = block_table[(size_t)(bt_rows ? bt_rows[seq] : seq) * bt_stride + j / page_size];
    const bool there = pg >= 0 && pg < num_pages;
    const bf16* src = pages + ((size_t)(there ? pg : 0) * page_size + j % page_size) * ROW;
    if (vec) {
        for (int e = lane * 8; e < ROW; e += 256)
            *reinterpret_cast<uint4*>(dst + e) = there ? *reinterpret_cast<const uint4*>(src + e) : make_uint4(0, 0, 0, 0);
    } else {
        for (int e = lane; e < ROW; e += 32) dst[e] = there ? src[e] : from_f32<bf16>(0.f);
    }
}

ACV_API int acv_latent_context(const void* pages, const int* page_seq, const int* page_idx, const int* kv_len,
                               const int* block_table, int bt_stride, const int* bt_rows, void* out, int n_pages, int ROW,
                               int page_size, int num_pages, cudaStream_t stream) {
    if (n_pages <= 0) return 0;
    if (ROW <= 0 || page_size <= 0 || num_pages <= 0) return ACV_ERR_SIZE;
    const int vec = ROW % 8 == 0 && !((uintptr_t)pages & 15) && !((uintptr_t)out & 15);
    acv_launch(PDL_MISC, latent_context_kernel, dim3(n_pages, LX_PAGE / 8), 256, 0, stream, (const bf16*)pages, page_seq, page_idx,
               kv_len, block_table, bt_stride, bt_rows, (bf16*)out, ROW, page_size, num_pages, vec);
    return acv_launch_status();
}

// E neighbouring elements (8: 16 bytes) at a time
template <int E>
struct LxPiece { bf16 x[E]; };
template <> struct __align__(16) LxPiece<8> { bf16 x[8]; };

// grid (pages, H): a block writes a head's 128 key rows and 128 value rows of a page
template <int E>
__global__ void __launch_bounds__(256)
latent_pack_kernel(const bf16* __restrict__ kv, int ldkv, const bf16* __restrict__ rows, int ROW, bf16* __restrict__ kp,
                   bf16* __restrict__ vp, int H, int D, int R, int DV, int KR, int HD) {
    pdl_launch_dependents();
    pdl_wait();
    const int pg = blockIdx.x, h = blockIdx.y, per = HD / E;
    LxPiece<E> zero;
#pragma unroll
    for (int i = 0; i < E; ++i) zero.x[i] = from_f32<bf16>(0.f);
    for (int i = threadIdx.x; i < LX_PAGE * per; i += blockDim.x) {
        const int r = i / per, e = (i - r * per) * E;
        const size_t row = (size_t)pg * LX_PAGE + r, at = (((size_t)pg * H + h) * LX_PAGE + r) * HD + e;
        LxPiece<E> k = zero, v = zero;
        if (e < D) k = *reinterpret_cast<const LxPiece<E>*>(kv + row * ldkv + (size_t)h * D + e);
        else if (e < D + R) k = *reinterpret_cast<const LxPiece<E>*>(rows + row * ROW + KR + e - D);
        if (e < DV) v = *reinterpret_cast<const LxPiece<E>*>(kv + row * ldkv + (size_t)H * D + (size_t)h * DV + e);
        *reinterpret_cast<LxPiece<E>*>(kp + at) = k;
        *reinterpret_cast<LxPiece<E>*>(vp + at) = v;
    }
}

// kv: [n_pages * 128] rows of H*D + H*DV at ldkv; rows: the kept rows of acv_latent_context; kp, vp [n_pages][H][128][HD]
ACV_API int acv_latent_pack(const void* kv, int ldkv, const void* rows, int ROW, void* kp, void* vp, int n_pages, int H, int D,
                            int R, int DV, int KR, int HD, cudaStream_t stream) {
    if (n_pages <= 0) return 0;
    if (H <= 0 || H > 65535 || D < 0 || R <= 0 || DV <= 0 || D + R > HD || DV > HD || KR + R != ROW) return ACV_ERR_SIZE;
    const bool vec = D % 8 == 0 && R % 8 == 0 && DV % 8 == 0 && KR % 8 == 0 && HD % 8 == 0 && ldkv % 8 == 0 &&
                     !(((uintptr_t)kv | (uintptr_t)rows | (uintptr_t)kp | (uintptr_t)vp) & 15);
    const dim3 grid(n_pages, H);
    if (vec)
        acv_launch(PDL_MISC, latent_pack_kernel<8>, grid, 256, 0, stream, (const bf16*)kv, ldkv, (const bf16*)rows, ROW, (bf16*)kp,
                   (bf16*)vp, H, D, R, DV, KR, HD);
    else
        acv_launch(PDL_MISC, latent_pack_kernel<1>, grid, 256, 0, stream, (const bf16*)kv, ldkv, (const bf16*)rows, ROW, (bf16*)kp,
                   (bf16*)vp, H, D, R, DV, KR, HD);
    return acv_launch_status();
}

// q: rows of H heads of HD elements [plain (D) | rotated (R) | ...]; listed rows: plain parts to qd [n][H][D], rotated parts to
// met [n][H][KR + R] behind the place of the latent part.  A block a row.
__global__ void latent_pick_kernel(const bf16* __restrict__ q, int HD, const int* __restrict__ list, bf16* __restrict__ qd,
                                   bf16* __restrict__ met, int H, int D, int R, int KR) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x, W = D + R;
    const bf16* src = q + (size_t)list[i] * H * HD;
    for (int x = threadIdx.x; x < H * W; x += blockDim.x) {
        const int h = x / W, e = x - h * W;
        const bf16 v = src[(size_t)h * HD + e];
        if (e < D) qd[((size_t)i * H + h) * D + e] = v;
        else met[((size_t)i * H + h) * (KR + R) + KR + e - D] = v;
    }
}

ACV_API int acv_latent_pick(const void* q, int HD, const int* list, void* qd, void* met, int n, int H, int D, int R, int KR,
                            cudaStream_t stream) {
    if (n <= 0) return 0;
    if (H <= 0 || D < 0 || R <= 0 || KR <= 0 || D + R > HD) return ACV_ERR_SIZE;
    acv_launch(PDL_MISC, latent_pick_kernel, n, 256, 0, stream, (const bf16*)q, HD, list, (bf16*)qd, (bf16*)met, H, D, R, KR);
    return acv_launch_status();
}

// out[row][h DV + e] = x[i][h HD + e] * sigmoid(gate[row][h DV + e]), row = list[i] (or i); E elements a thread
template <int E>
__global__ void __launch_bounds__(256)
heads_gated_kernel(const bf16* __restrict__ x, int HD, const bf16* __restrict__ gate, int ldg, const int* __restrict__ list,
                   bf16* __restrict__ out, int ldo, int n, int H, int DV) {
    pdl_launch_dependents();
    pdl_wait();
    const int per = H * DV / E;
    const long long id = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const int i = (int)(id / per), c = (int)(id - (long long)i * per) * E;
    if (i >= n) return;
    const int h = c / DV, row = list ? list[i] : i;
    LxPiece<E> v = *reinterpret_cast<const LxPiece<E>*>(x + ((size_t)i * H + h) * HD + c - h * DV);
    if (gate) {
        const LxPiece<E> g = *reinterpret_cast<const LxPiece<E>*>(gate + (size_t)row * ldg + c);
#pragma unroll
        for (int e = 0; e < E; ++e) v.x[e] = from_f32<bf16>(to_f32(v.x[e]) * __fdividef(1.f, 1.f + __expf(-to_f32(g.x[e]))));
    }
    *reinterpret_cast<LxPiece<E>*>(out + (size_t)row * ldo + c) = v;
}

ACV_API int acv_heads_gated(const void* x, int HD, const void* gate, int ldg, const int* list, void* out, int ldo, int n, int H,
                            int DV, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (H <= 0 || DV <= 0 || DV > HD) return ACV_ERR_SIZE;
    const bool vec = DV % 8 == 0 && HD % 8 == 0 && ldo % 8 == 0 && (!gate || (ldg % 8 == 0 && !((uintptr_t)gate & 15))) &&
                     !(((uintptr_t)x | (uintptr_t)out) & 15);
    const long long threads = (long long)n * H * DV / (vec ? 8 : 1);
    const int grid = (int)((threads + 255) / 256);
    if (vec)
        acv_launch(PDL_MISC, heads_gated_kernel<8>, grid, 256, 0, stream, (const bf16*)x, HD, (const bf16*)gate, ldg, list,
                   (bf16*)out, ldo, n, H, DV);
    else
        acv_launch(PDL_MISC, heads_gated_kernel<1>, grid, 256, 0, stream, (const bf16*)x, HD, (const bf16*)gate, ldg, list,
                   (bf16*)out, ldo, n, H, DV);
    return acv_launch_status();
}
