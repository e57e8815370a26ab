// Linear attention with one constant decay a head, for prompts, in bfloat16 on the tensor cores (mma.sync m16n8k16, fp32
// accumulation): the recurrence
//   S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// taken 64 tokens at a time.  With S the state before a chunk of n tokens, t and s counting inside it:
//   o_t = d^(t+1) S^T q_t + sum_{s <= t} d^(t-s) (q_t . k_s) v_s
//   S  <- d^n S + sum_s k_s (d^(n-1-s) v_s)^T
// Every exponent is >= 0 and the powers come from a table [heads][65] (float32, made from the decay in double precision),
// so nothing over- or underflows however strong the decay.
//
// q, k and v are the activations SiLU(row) rounded to bf16, as the projections' activations are elsewhere.  What the
// products take that is not such an activation (the chunk's weights d^(t-s) q.k, the state where it is read, the
// decayed values) goes in as two bf16 terms, x = hi + lo with hi = bf16(x) and lo = bf16(x - hi), so that it keeps 16
// bits; the state itself is fp32 in registers from chunk to chunk and in the cache.
//
// One block per (sequence, head, 64 value columns, segment): 4 warps, each with a quarter of the state's rows and 16 of
// the chunk's tokens.  Long prompts are cut into segments that run side by side, in three passes as in recurrent.cu: each
// segment's own contribution from zero (LOCAL), the state at every segment's start (decay_combine_kernel), and the walk
// that writes o (FINAL; WHOLE where there is one segment).
#include "common.cuh"

namespace {

constexpr int NT = 128, C = 64, PT = 64;
constexpr int LDV = PT + 8;                            // padded rows: ldmatrix without bank conflicts
constexpr int POW_N = C + 1;
constexpr int PASS_WHOLE = 0, PASS_LOCAL = 1, PASS_FINAL = 2;

struct Args {
    const bf16 *q, *k, *v;                             // [T, H * N], [T, H * N], [T, H * P]
    long ldq, ldk, ldv;
    const float* powers;                               // [H][65]: d^0 .. d^64
    float* state;                                      // [slot][H][N][P]
    long state_stride;
    float* y;                                          // [T, H * P]
    long ldy;
    const int *seq_start, *seq_slot;
    int n_seqs, H, N, P, seg_len, max_segs, silu;
    float* seg_state;                                  // [seq][segment][H][N][P]
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t bits(__nv_bfloat162 h) { return *reinterpret_cast<uint32_t*>(&h); }
// two floats as bf16 pairs hi + lo
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = bits(h);
    lo = bits(__floats2bfloat162_rn(a - __low2float(h), b - __high2float(h)));
}
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + __expf(-x)); }

// eight activations of a row: SiLU where asked for, rounded to bf16
__device__ __forceinline__ uint4 act8(uint4 raw, bool silu) {
    if (!silu) return raw;
    uint32_t* w = reinterpret_cast<uint32_t*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(w + i);
        w[i] = bits(__floats2bfloat162_rn(silu_f(__low2float(h)), silu_f(__high2float(h))));
    }
    return raw;
}

template <int NP> constexpr size_t smem_bytes() {
    return (size_t)(2 * C * (NP + 8) + 3 * C * LDV + 2 * NP * LDV) * sizeof(bf16) + (POW_N + 3) / 4 * 4 * sizeof(float);
}

template <int NP, int PASS>
__global__ void __launch_bounds__(NT, 2) decay_chunk_kernel(const Args a) {
    constexpr int LDK = NP + 8, MT = NP / 64, KS = NP / 16;
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);      // [C][LDK]
    bf16* Ks = Qs + C * LDK;                           // [C][LDK]
    bf16* Vs = Ks + C * LDK;                           // [C][LDV]: v
    bf16* Vhi = Vs + C * LDV;                          // [C][LDV]: d^(n-1-s) v in two terms
    bf16* Vlo = Vhi + C * LDV;
    bf16* Shi = Vlo + C * LDV;                         // [NP][LDV]: the state in two terms
    bf16* Slo = Shi + NP * LDV;
    float* pw = reinterpret_cast<float*>(Slo + NP * LDV);      // [65]
    pdl_launch_dependents();
    const int ptiles = (a.P + PT - 1) / PT;
    int bid = blockIdx.x;
    const int p0 = (bid % ptiles) * PT;
    bid /= ptiles;
    const int h = bid % a.H, b = bid / a.H, seg = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int N = a.N, P = a.P;
    for (int i = threadIdx.x; i < POW_N; i += NT) pw[i] = a.powers[h * POW_N + i];
    pdl_wait();
    const int s0 = a.seq_start[b], s1 = a.seq_start[b + 1];
    const int n_segs = PASS == PASS_WHOLE ? 1 : (s1 - s0 + a.seg_len - 1) / a.seg_len;
    if (PASS == PASS_LOCAL ? seg >= n_segs - 1 : PASS == PASS_FINAL ? seg >= n_segs : s1 <= s0) return;
    const int t0 = PASS == PASS_WHOLE ? s0 : s0 + seg * a.seg_len;
    const int t1 = PASS == PASS_WHOLE ? s1 : min(s1, t0 + a.seg_len);
    float* st = a.state + (long)a.seq_slot[b] * a.state_stride + (long)h * N * P;
    float* sg = PASS == PASS_WHOLE ? nullptr : a.seg_state + (((long)b * a.max_segs + seg) * a.H + h) * N * P;
    const float* init = PASS == PASS_WHOLE ? st : PASS == PASS_FINAL ? sg : nullptr;

    // this warp's rows of the state: n = warp * NP / 4 + 16 mt + lane / 4 (+ 8), columns p0 + 8 j + 2 (lane % 4) (+ 1)
    const int nr = warp * (NP / 4) + (lane >> 2), pc = (lane & 3) * 2;
    float S[MT][PT / 8][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < PT / 8; ++j)
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                const int n = nr + mt * 16 + hi * 8, p = p0 + j * 8 + pc;
                float2 x = make_float2(0.f, 0.f);
                if (init && n < N && p < P) x = *reinterpret_cast<const float2*>(init + (long)n * P + p);
                S[mt][j][2 * hi] = x.x;
                S[mt][j][2 * hi + 1] = x.y;
            }

    const bool silu = a.silu;
    const int l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    for (int base = t0; base < t1; base += C) {
        const int n = min(C, t1 - base);               // tokens of this chunk
        __syncthreads();                               // the chunk before has been read
        const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll 4
        for (int idx = threadIdx.x; idx < C * (NP / 8); idx += NT) {
            const int r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
            const bool in = r < n && c < N;
            const uint4 kr = in ? *reinterpret_cast<const uint4*>(a.k + (long)(base + r) * a.ldk + (long)h * N + c) : zero;
            if (PASS != PASS_LOCAL) {
                const uint4 qr = in ? *reinterpret_cast<const uint4*>(a.q + (long)(base + r) * a.ldq + (long)h * N + c) : zero;
                *reinterpret_cast<uint4*>(Qs + r * LDK + c) = act8(qr, silu);
            }
            *reinterpret_cast<uint4*>(Ks + r * LDK + c) = act8(kr, silu);
        }
#pragma unroll
        for (int idx = threadIdx.x; idx < C * (PT / 8); idx += NT) {
            const int r = idx / (PT / 8), c = (idx % (PT / 8)) * 8;
            const bool in = r < n && p0 + c < P;
            uint4 vr = in ? *reinterpret_cast<const uint4*>(a.v + (long)(base + r) * a.ldv + (long)h * P + p0 + c) : zero;
            vr = act8(vr, silu);
            if (PASS != PASS_LOCAL) *reinterpret_cast<uint4*>(Vs + r * LDV + c) = vr;
            const float g = r < n ? pw[n - 1 - r] : 0.f;
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(reinterpret_cast<const uint32_t*>(&vr) + i);
                split2(g * __low2float(x), g * __high2float(x), hi[i], lo[i]);
            }
            *reinterpret_cast<uint4*>(Vhi + r * LDV + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(Vlo + r * LDV + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        if (PASS != PASS_LOCAL) {
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int j = 0; j < PT / 8; ++j)
#pragma unroll
                    for (int hi = 0; hi < 2; ++hi) {
                        uint32_t xh, xl;
                        split2(S[mt][j][2 * hi], S[mt][j][2 * hi + 1], xh, xl);
                        const int at = (nr + mt * 16 + hi * 8) * LDV + j * 8 + pc;
                        *reinterpret_cast<uint32_t*>(Shi + at) = xh;
                        *reinterpret_cast<uint32_t*>(Slo + at) = xl;
                    }
        }
        __syncthreads();
        if (PASS != PASS_LOCAL && warp * 16 < n) {
            // this warp's 16 tokens: rows warp * 16 + lane / 4 (+ 8)
            const int tl = warp * 16 + (lane >> 2);
            uint32_t qa[KS][4];
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) ldsm_x4(qa[ks], smem_u32(Qs + (warp * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8));
            float o[PT / 8][4];
#pragma unroll
            for (int j = 0; j < PT / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {          // S^T q: what comes from the chunks before
#pragma unroll
                for (int j = 0; j < PT / 8; j += 2) {
                    uint32_t bh[4], bl[4];
                    const int at = (ks * 16 + l7 + b3 * 8) * LDV + j * 8 + b4 * 8;
                    ldsm_x4_t(bh, smem_u32(Shi + at));
                    ldsm_x4_t(bl, smem_u32(Slo + at));
                    mma_bf16(o[j], qa[ks], bh[0], bh[1]);
                    mma_bf16(o[j + 1], qa[ks], bh[2], bh[3]);
                    mma_bf16(o[j], qa[ks], bl[0], bl[1]);
                    mma_bf16(o[j + 1], qa[ks], bl[2], bl[3]);
                }
            }
            const float dlo = pw[tl + 1], dhi = pw[tl + 9];
#pragma unroll
            for (int j = 0; j < PT / 8; ++j) {
                o[j][0] *= dlo; o[j][1] *= dlo;
                o[j][2] *= dhi; o[j][3] *= dhi;
            }
#pragma unroll 1
            for (int kb = 0; kb <= warp; ++kb) {       // the chunk's own keys, 16 at a time
                float w[2][4];
#pragma unroll
                for (int i = 0; i < 2; ++i) w[i][0] = w[i][1] = w[i][2] = w[i][3] = 0.f;
#pragma unroll
                for (int ks = 0; ks < KS; ++ks) {
                    uint32_t kf[4];
                    ldsm_x4(kf, smem_u32(Ks + (kb * 16 + l7 + b4 * 8) * LDK + ks * 16 + b3 * 8));
                    mma_bf16(w[0], qa[ks], kf[0], kf[1]);
                    mma_bf16(w[1], qa[ks], kf[2], kf[3]);
                }
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int dist = tl + (e >> 1) * 8 - (kb * 16 + i * 8 + pc + (e & 1));
                        w[i][e] = dist >= 0 ? w[i][e] * pw[dist] : 0.f;
                    }
                uint32_t ah[4], al[4];
                split2(w[0][0], w[0][1], ah[0], al[0]);
                split2(w[0][2], w[0][3], ah[1], al[1]);
                split2(w[1][0], w[1][1], ah[2], al[2]);
                split2(w[1][2], w[1][3], ah[3], al[3]);
#pragma unroll
                for (int j = 0; j < PT / 8; j += 2) {
                    uint32_t vf[4];
                    ldsm_x4_t(vf, smem_u32(Vs + (kb * 16 + l7 + b3 * 8) * LDV + j * 8 + b4 * 8));
                    mma_bf16(o[j], ah, vf[0], vf[1]);
                    mma_bf16(o[j + 1], ah, vf[2], vf[3]);
                    mma_bf16(o[j], al, vf[0], vf[1]);
                    mma_bf16(o[j + 1], al, vf[2], vf[3]);
                }
            }
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                const int t = tl + hi * 8;
                if (t >= n) continue;
                float* yr = a.y + (long)(base + t) * a.ldy + (long)h * P + p0 + pc;
#pragma unroll
                for (int j = 0; j < PT / 8; ++j)
                    if (p0 + j * 8 < P) *reinterpret_cast<float2*>(yr + j * 8) = make_float2(o[j][2 * hi], o[j][2 * hi + 1]);
            }
        }
        // the state: d^n S + K^T (decayed V)
        const float dn = pw[n];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int j = 0; j < PT / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[mt][j][e] *= dn;
#pragma unroll
        for (int sb = 0; sb < C / 16; ++sb) {
            if (sb * 16 >= n) break;
            uint32_t ka[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
                ldsm_x4_t(ka[mt], smem_u32(Ks + (sb * 16 + b4 * 8 + l7) * LDK + warp * (NP / 4) + mt * 16 + b3 * 8));
#pragma unroll
            for (int j = 0; j < PT / 8; j += 2) {
                uint32_t vh[4], vl[4];
                const int at = (sb * 16 + l7 + b3 * 8) * LDV + j * 8 + b4 * 8;
                ldsm_x4_t(vh, smem_u32(Vhi + at));
                ldsm_x4_t(vl, smem_u32(Vlo + at));
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mma_bf16(S[mt][j], ka[mt], vh[0], vh[1]);
                    mma_bf16(S[mt][j + 1], ka[mt], vh[2], vh[3]);
                    mma_bf16(S[mt][j], ka[mt], vl[0], vl[1]);
                    mma_bf16(S[mt][j + 1], ka[mt], vl[2], vl[3]);
                }
            }
        }
    }
    float* dst = PASS == PASS_LOCAL ? sg : (PASS == PASS_WHOLE || seg == n_segs - 1) ? st : nullptr;
    if (dst) {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int j = 0; j < PT / 8; ++j)
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    const int n = nr + mt * 16 + hi * 8, p = p0 + j * 8 + pc;
                    if (n < N && p < P)
                        *reinterpret_cast<float2*>(dst + (long)n * P + p) = make_float2(S[mt][j][2 * hi], S[mt][j][2 * hi + 1]);
                }
    }
}

// The state at the start of every segment, from the cache's state and the segments' own contributions:
// S_in[0] = state, S_in[c + 1] = d^seg_len S_in[c] + local[c].  Four elements a thread; S_in[c] takes local[c]'s place.
__global__ void decay_combine_kernel(const Args a) {
    pdl_launch_dependents();
    pdl_wait();
    const long per_seq = (long)a.H * a.N * a.P;
    const long idx = ((long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (idx >= per_seq * a.n_seqs) return;
    const int b = (int)(idx / per_seq);
    const long e = idx % per_seq;
    const int h = (int)(e / ((long)a.N * a.P));
    const int len = a.seq_start[b + 1] - a.seq_start[b];
    const int n_segs = (len + a.seg_len - 1) / a.seg_len;
    double dd = 1.0;
    const double d64 = (double)a.powers[h * POW_N + C];
    for (int i = 0; i < a.seg_len / C; ++i) dd *= d64;
    const float d = (float)dd;
    float4 S = *reinterpret_cast<const float4*>(a.state + (long)a.seq_slot[b] * a.state_stride + e);
    float* sg = a.seg_state + (long)b * a.max_segs * per_seq + e;
    for (int c0 = 0; c0 < n_segs; c0 += 8) {           // eight segments' values are asked for at once, then chained
        float4 local[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
            local[i] = c0 + i < n_segs - 1 ? *reinterpret_cast<const float4*>(sg + (long)(c0 + i) * per_seq)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (c0 + i >= n_segs) break;
            *reinterpret_cast<float4*>(sg + (long)(c0 + i) * per_seq) = S;
            S = make_float4(fmaf(d, S.x, local[i].x), fmaf(d, S.y, local[i].y), fmaf(d, S.z, local[i].z), fmaf(d, S.w, local[i].w));
        }
    }
}

template <int NP>
int launch(const Args& a, cudaStream_t stream) {
    static bool configured = false;
    constexpr size_t smem = smem_bytes<NP>();
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_WHOLE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_LOCAL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_FINAL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const unsigned blocks = (unsigned)((long)a.n_seqs * a.H * ((a.P + PT - 1) / PT));
    if (a.max_segs <= 1) return plm_status_of(launch_pdl(decay_chunk_kernel<NP, PASS_WHOLE>, dim3(blocks), dim3(NT), smem, stream, a));
    cudaError_t e = launch_pdl(decay_chunk_kernel<NP, PASS_LOCAL>, dim3(blocks, a.max_segs - 1), dim3(NT), smem, stream, a);
    if (e != cudaSuccess) return (int)e;
    const long quads = (long)a.n_seqs * a.H * a.N * a.P / 4;
    e = launch_pdl(decay_combine_kernel, dim3((unsigned)((quads + 127) / 128)), dim3(128), 0, stream, a);
    if (e != cudaSuccess) return (int)e;
    return plm_status_of(launch_pdl(decay_chunk_kernel<NP, PASS_FINAL>, dim3(blocks, a.max_segs), dim3(NT), smem, stream, a));
}

}  // namespace

// How a step of `n_tokens` tokens whose longest sequence brings `max_new` of them is cut: out[0] tokens per segment (a
// multiple of 64), out[1] segments of the longest sequence (1: one pass, no scratch memory): as many as make one wave of
// blocks at two an SM, each of at least 128 tokens, and no more than keep the scratch memory under 1 GiB.
extern "C" int plm_decay_chunk_plan(int n_seqs, int H, int N, int P, int max_new, int n_tokens, int* out) {
    out[0] = max_new > 0 ? (max_new + C - 1) / C * C : C;
    out[1] = 1;
    if (n_seqs <= 0 || H <= 0 || N <= 0 || P <= 0) return PLM_ERR_SHAPE;
    if (max_new < 4 * C) return PLM_OK;
    long busy = n_tokens > 0 ? ((long)n_tokens + max_new - 1) / max_new : n_seqs;     // sequences' worth of work
    if (busy > n_seqs) busy = n_seqs;
    if (busy < 1) busy = 1;
    const long blocks = busy * H * ((P + PT - 1) / PT);
    long segs = 2L * PLM_SM_COUNT / blocks;
    if (segs > max_new / (2 * C)) segs = max_new / (2 * C);
    const long state_bytes = (long)n_seqs * H * N * P * 4;
    while (segs > 1 && segs * state_bytes > (1L << 30)) --segs;
    if (segs <= 1) return PLM_OK;
    const int len = (int)(((max_new + segs - 1) / segs + C - 1) / C * C);
    out[0] = len;
    out[1] = (max_new + len - 1) / len;
    return PLM_OK;
}

// q, k [T, H * N], v [T, H * P] bf16 with row strides (N a multiple of 16 up to 128, P of 8, rows on 16-byte boundaries);
// powers [H][65] fp32; state [slots][>= H * N * P] fp32; y [T, H * P] fp32; seg_state for max_segs > 1.
extern "C" int plm_decay_chunk_scan(const void* q, const void* k, const void* v, long ldq, long ldk, long ldv, const float* powers,
                                    float* state, long state_stride, float* y, long ldy, const int* seq_start,
                                    const int* seq_slot, int n_seqs, int H, int N, int P, int seg_len, int max_segs,
                                    float* seg_state, int silu, cudaStream_t stream) {
    if (n_seqs <= 0 || H <= 0 || N <= 0 || P <= 0 || N % 16 || N > 128 || P % 8) return PLM_ERR_SHAPE;
    if (max_segs > 1 && (!seg_state || seg_len <= 0 || seg_len % C || max_segs > 65535)) return PLM_ERR_SHAPE;
    if ((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)y | (uintptr_t)seg_state) & 15) || ldq % 8 ||
        ldk % 8 || ldv % 8 || state_stride % 4 || ldy % 4)
        return PLM_ERR_ALIGN;
    Args a;
    a.q = (const bf16*)q, a.k = (const bf16*)k, a.v = (const bf16*)v;
    a.ldq = ldq, a.ldk = ldk, a.ldv = ldv;
    a.powers = powers, a.state = state, a.state_stride = state_stride, a.y = y, a.ldy = ldy;
    a.seq_start = seq_start, a.seq_slot = seq_slot;
    a.n_seqs = n_seqs, a.H = H, a.N = N, a.P = P, a.seg_len = seg_len, a.max_segs = max_segs < 1 ? 1 : max_segs;
    a.silu = silu, a.seg_state = seg_state;
    return N <= 64 ? launch<64>(a, stream) : launch<128>(a, stream);
}
