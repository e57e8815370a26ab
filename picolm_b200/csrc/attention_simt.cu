// Causal attention of new tokens over the paged cache, one warp per
// (token, query head), on the CUDA cores with fp32 arithmetic throughout.
//
// For a query at absolute position p with head h, KV head g = h / (H / G):
//   s_t = (q_h . K[t, g]) * scale  for t in [lo, p],  out_h = softmax(s) . V[:, g]
// with the running (max, sum, acc) update of the reference's `attn_core`
// (picolm/model_attention.c:43-140; max starts at -1e30, causal by the loop
// bound) taken 32 keys at a time.  lo = 0, or p - window + 1 for a sliding
// window, or the start of p's chunk for a mask of chunks (plm_first_key); with `keep` > 0 the positions before
// min(keep, lo) are seen too; with `slopes` [H] a score loses slopes[h] * (p - t).  Keys and values of position t of sequence b live at
//   cache[block_table[b][t / PLM_PAGE]][g][t % PLM_PAGE][0..hd)
// and the new tokens' own K/V are already there when this kernel runs.
//
// This is the attention of the float32 path, and the any-size attention of the
// bfloat16 path (head sizes that the tensor-core kernels refuse).  A row's
// result depends on its own position and sequence only.
#include "common.cuh"

namespace {

constexpr int WARPS = 4;
constexpr int MAX_HD = 1024;           // the largest head size; acc registers per lane: MAX_HD / 32 of the instance

// MAX_HD: the instance's largest head size (256 for the usual heads; 512 and 1024 for the wide single head of a
// latent cache, whose keys are the latents themselves).
template <typename Ta, typename Tc, int MAX_HD>
__global__ void __launch_bounds__(WARPS * 32)
attention_rows_kernel(const Ta* q, const Tc* kc, const Tc* vc,
                      Ta* __restrict__ out, const int* tok_pos, const int* tok_seq,
                      const int* block_table, int max_pages, int H, int G, int hd, float scale,
                      int window, const float* sink, int keep, const float* slopes) {
    extern __shared__ float q_sm[];                 // [WARPS][hd]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x;
    const int h = blockIdx.y * WARPS + warp;
    if (h >= H) return;                             // warp-level exit; no block barrier below
    const int g = h / (H / G);
    const int pos = PLM_POSITION(tok_pos[t]);
    const int* pages = block_table + (size_t)PLM_SEQ_NO(tok_seq[t]) * max_pages;
    float* qs = q_sm + warp * hd;
    const Ta* qrow = q + ((size_t)t * H + h) * hd;
    for (int i = lane; i < hd; i += 32) qs[i] = to_f32<Ta>(qrow[i]);
    __syncwarp();

    float acc[MAX_HD / 32];
#pragma unroll
    for (int i = 0; i < MAX_HD / 32; ++i) acc[i] = 0.f;
    float m = -1e30f, l = 0.f;
    const int lo = plm_first_key(pos, window);
    const int n_kept = min(keep, lo);               // kept first positions in front of the window
    const int n_keys_all = n_kept + pos - lo + 1;
    const int skip = lo - n_kept;                   // the n-th key this row sees: n, or n + skip from n_kept on
    const float slope = slopes ? slopes[h] : 0.f;

    for (int base = 0; base < n_keys_all; base += 32) {
        const int nth = base + lane;
        const int key = nth < n_kept ? nth : nth + skip;
        float s = -1e30f;
        const bool valid = nth < n_keys_all;
        if (valid) {
            const int page = PLM_PAGE_NO(pages[key / PLM_PAGE]);
            const Tc* kr = kc + (((size_t)page * G + g) * PLM_PAGE + key % PLM_PAGE) * hd;
            float dot = 0.f;
            for (int i = 0; i < hd; ++i) dot = fmaf(qs[i], to_f32<Tc>(kr[i]), dot);
            s = dot * scale;
            if (slopes) s -= slope * (float)(pos - key);
        }
        const float m_new = fmaxf(m, warp_max(s));
        const float corr = expf(m - m_new);
        const float p = valid ? expf(s - m_new) : 0.f;
        l = l * corr + warp_sum(p);
#pragma unroll
        for (int i = 0; i < MAX_HD / 32; ++i) acc[i] *= corr;
        const int n_keys = min(32, n_keys_all - base);
        for (int j = 0; j < n_keys; ++j) {
            const float pj = __shfl_sync(0xffffffffu, p, j);
            const int kj = base + j < n_kept ? base + j : base + j + skip;
            const int page = PLM_PAGE_NO(pages[kj / PLM_PAGE]);
            const Tc* vr = vc + (((size_t)page * G + g) * PLM_PAGE + kj % PLM_PAGE) * hd;
#pragma unroll
            for (int i = 0; i < MAX_HD / 32; ++i) {
                const int d = lane + 32 * i;
                if (d < hd) acc[i] = fmaf(pj, to_f32<Tc>(vr[d]), acc[i]);
            }
        }
        m = m_new;
    }
    if (sink) {
        // a sink: one more term exp(sink[h]) in the denominator, with no key and no value, not scaled
        const float sk = sink[h], m_new = fmaxf(m, sk);
        const float corr = expf(m - m_new);
        l = l * corr + expf(sk - m_new);
#pragma unroll
        for (int i = 0; i < MAX_HD / 32; ++i) acc[i] *= corr;
    }
    const float inv = 1.0f / l;
    Ta* o = out + ((size_t)t * H + h) * hd;
#pragma unroll
    for (int i = 0; i < MAX_HD / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < hd) o[d] = from_f32<Ta>(acc[i] * inv);
    }
}

}  // namespace

// q [T, H, hd] and out [T, H, hd] have the activation type, the cache its own;
// both are PLM_F32 or both PLM_BF16.
extern "C" int plm_attention_rows(const void* q, const void* kc, const void* vc, void* out, int dtype,
                                  const int* tok_pos, const int* tok_seq, const int* block_table, int max_pages,
                                  int n_tokens, int H, int G, int hd, float scale, int window, const float* sink,
                                  int keep, const float* slopes, cudaStream_t stream) {
    if (n_tokens <= 0) return PLM_OK;
    if (H <= 0 || G <= 0 || H % G || hd <= 0 || hd > MAX_HD || keep < 0) return PLM_ERR_SHAPE;
    dim3 grid(n_tokens, (H + WARPS - 1) / WARPS);
    const size_t smem = (size_t)WARPS * hd * sizeof(float);
#define ROWS_LAUNCH(Ta_, MAXHD_)                                                                                       \
    attention_rows_kernel<Ta_, Ta_, MAXHD_><<<grid, WARPS * 32, smem, stream>>>(                                       \
        (const Ta_*)q, (const Ta_*)kc, (const Ta_*)vc, (Ta_*)out, tok_pos, tok_seq, block_table, max_pages, H, G, hd, \
        scale, window, sink, keep, slopes)
#define ROWS_BY_SIZE(Ta_)                          \
    do {                                           \
        if (hd <= 256) ROWS_LAUNCH(Ta_, 256);      \
        else if (hd <= 512) ROWS_LAUNCH(Ta_, 512); \
        else ROWS_LAUNCH(Ta_, 1024);               \
    } while (0)
    if (dtype == PLM_F32)
        ROWS_BY_SIZE(float);
    else if (dtype == PLM_BF16)
        ROWS_BY_SIZE(bf16);
    else
        return PLM_ERR_DTYPE;
#undef ROWS_BY_SIZE
#undef ROWS_LAUNCH
    return plm_launch_status();
}
