// The delta rule with one decay a head, for prompts, on the tensor cores (mma.sync m16n8k16, fp32 sums): the recurrence
//   S <- g_t S,  u_t = beta_t (v_t - S^T k_t),  S <- S + k_t u_t^T,  o_t = S^T q_t
// taken 64 tokens at a time.  With S the state before a chunk, L_t the running sum of log g inside it and C its last token,
//   u_t = beta_t (v_t - e^(L_t) S^T k_t) - sum_{s<t} A_ts u_s,   A_ts = beta_t e^(L_t - L_s) (k_t . k_s)
// is a unit lower triangular system whose right side is linear in S, so
//   U = U0 - W S,   (1 + A) U0 = (beta_t v_t),   (1 + A) W = (beta_t e^(L_t) k_t)
//   O = (e^(L_t) q_t) S + M U,   M_ts = e^(L_t - L_s) (q_t . k_s), s <= t
//   S <- e^(L_C) S + sum_s (e^(L_C - L_s) k_s) u_s^T
// Every exponent is <= 0, so no choice of decays overflows.  A first kernel makes what does not depend on the state (U0, W,
// M, the scaled q and k) for all chunks side by side; both systems are solved in fp32 by forward substitution, a thread a
// column with its 64 unknowns in registers.  A second kernel walks a sequence's chunks with the state in registers.
//
// Whatever a product takes goes in as two bf16 terms (mma_common.cuh; hi hi + hi lo + lo hi), the state itself stays fp32.
// The first kernel leaves its matrices in the order of the second one's A fragments (16 bytes a lane), so that each warp of
// the walk loads the rows it owns straight into registers, a phase ahead of their use.
#include "mma_common.cuh"

namespace {

constexpr int NT = 256, C = 64, PT = 32;
constexpr int LDS_ = PT + 8;                           // padded rows: ldmatrix without bank conflicts
constexpr int LDA = C + 4;                             // rows of A^T

// The workspace of one (chunk, head), in bytes: W | Q | K^T | M as fragments, each tile 512 bytes, its two terms one behind
// the other; then U0 [C][P] fp32 and e^(L_C).
template <int NP> struct Layout {
    static constexpr int KS = NP / 16;
    static constexpr long W = 0, Q = W + 4L * KS * 1024, K = Q + 4L * KS * 1024, M = K + 4L * KS * 1024, U0 = M + 16L * 1024;
    __host__ __device__ static long bytes(int P) { return U0 + (long)C * P * 4 + 16; }
};

__device__ __forceinline__ void put_tile(uint8_t* tile, int lane, const uint32_t (&hi)[4], const uint32_t (&lo)[4]) {
    reinterpret_cast<uint4*>(tile)[lane] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    reinterpret_cast<uint4*>(tile)[32 + lane] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
}

template <int NP> constexpr size_t prep_smem() {
    return (size_t)4 * C * (NP + 8) * sizeof(bf16) + (size_t)C * LDA * sizeof(float) + 3 * C * sizeof(float);
}

// grid (chunk of the sequence, sequence, head)
template <int NP>
__global__ void __launch_bounds__(NT, 2)
delta_head_prep_kernel(const float* qn, const float* kn, const float* lgd, const float* beta, const bf16* v, long ldv,
                       uint8_t* __restrict__ ws, const int* seq_start, int H, int N, int P, int heads_per_group) {
    constexpr int LDK = NP + 8, KS = NP / 16;
    using Lay = Layout<NP>;
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* Kh = reinterpret_cast<bf16*>(smem_raw);      // [C][LDK] each: k and q in two terms; then W in the place of q
    bf16* Kl = Kh + C * LDK;
    bf16* Qh = Kl + C * LDK;
    bf16* Ql = Qh + C * LDK;
    float* At = reinterpret_cast<float*>(Ql + C * LDK);    // [s][t]
    float* L = At + C * LDA;                           // [C] running sums
    float* eL = L + C;                                 // [C] their exponentials
    float* bt = eL + C;                                // [C] beta, 0 behind the last token
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x, b = blockIdx.y, h = blockIdx.z;
    const int s0 = seq_start[b], s1 = seq_start[b + 1];
    const int t0 = s0 + c * C;
    if (t0 >= s1) return;
    const int n = min(C, s1 - t0);
    const int G = H / heads_per_group, g = h / heads_per_group;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    uint8_t* out = ws + ((long)(s0 / C + b + c) * H + h) * Lay::bytes(P);
    for (int idx = threadIdx.x; idx < C * (NP / 2); idx += NT) {
        const int r = idx / (NP / 2), i = (idx % (NP / 2)) * 2;
        float2 q = make_float2(0.f, 0.f), k = q;
        if (r < n && i < N) {                          // (N is a multiple of 16)
            const long at = ((long)(t0 + r) * G + g) * N + i;
            q = *reinterpret_cast<const float2*>(qn + at);
            k = *reinterpret_cast<const float2*>(kn + at);
        }
        split2(q.x, q.y, *reinterpret_cast<uint32_t*>(Qh + r * LDK + i), *reinterpret_cast<uint32_t*>(Ql + r * LDK + i));
        split2(k.x, k.y, *reinterpret_cast<uint32_t*>(Kh + r * LDK + i), *reinterpret_cast<uint32_t*>(Kl + r * LDK + i));
    }
    if (warp == 0) {
        // two logarithms a lane, their sums along the warp
        const float a = 2 * lane < n ? lgd[(long)(t0 + 2 * lane) * H + h] : 0.f;
        const float d = 2 * lane + 1 < n ? lgd[(long)(t0 + 2 * lane + 1) * H + h] : 0.f;
        float run = a + d;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        const float before = __shfl_up_sync(0xffffffffu, run, 1);
        const float l0 = (lane ? before : 0.f) + a, l1 = l0 + d;
        L[2 * lane] = l0, L[2 * lane + 1] = l1;
        eL[2 * lane] = expf(l0), eL[2 * lane + 1] = expf(l1);
    }
    if (threadIdx.x < C) bt[threadIdx.x] = threadIdx.x < n ? beta[(long)(t0 + threadIdx.x) * H + h] : 0.f;
    __syncthreads();
    const int g8 = lane >> 2, pc = (lane & 3) * 2, l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    const float lend = L[C - 1];
    {
        // warps 0..3: A of sixteen tokens, 4..7: M; key tiles up to the diagonal
        const int i = warp & 3;
        const bf16 *Xh = warp < 4 ? Kh : Qh, *Xl = warp < 4 ? Kl : Ql;
        float w[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) w[j][0] = w[j][1] = w[j][2] = w[j][3] = 0.f;
#pragma unroll 2
        for (int ks = 0; ks < KS; ++ks) {
            uint32_t xh[4], xl[4];
            const int at = (i * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8;
            ldsm_x4(xh, smem_u32(Xh + at));
            ldsm_x4(xl, smem_u32(Xl + at));
#pragma unroll
            for (int kb = 0; kb < 4; ++kb) {
                if (kb > i) break;
                uint32_t kh[4], kl[4];
                const int ka = (kb * 16 + l7 + b4 * 8) * LDK + ks * 16 + b3 * 8;
                ldsm_x4(kh, smem_u32(Kh + ka));
                ldsm_x4(kl, smem_u32(Kl + ka));
                mma_bf16(w[2 * kb], xh, kh[0], kh[1]);
                mma_bf16(w[2 * kb + 1], xh, kh[2], kh[3]);
                mma_bf16(w[2 * kb], xh, kl[0], kl[1]);
                mma_bf16(w[2 * kb + 1], xh, kl[2], kl[3]);
                mma_bf16(w[2 * kb], xl, kh[0], kh[1]);
                mma_bf16(w[2 * kb + 1], xl, kh[2], kh[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = i * 16 + g8 + (e >> 1) * 8, s = j * 8 + pc + (e & 1);
                if (warp < 4)
                    At[s * LDA + t] = s < t ? bt[t] * w[j][e] * expf(L[t] - L[s]) : 0.f;
                else
                    w[j][e] = s <= t ? w[j][e] * expf(L[t] - L[s]) : 0.f;
            }
        if (warp >= 4) {
#pragma unroll
            for (int kb = 0; kb < 4; ++kb) {
                if (kb > i) break;                     // (the walk does not read the tiles behind the diagonal)
                uint32_t hi[4], lo[4];
                split2(w[2 * kb][0], w[2 * kb][1], hi[0], lo[0]);
                split2(w[2 * kb][2], w[2 * kb][3], hi[1], lo[1]);
                split2(w[2 * kb + 1][0], w[2 * kb + 1][1], hi[2], lo[2]);
                split2(w[2 * kb + 1][2], w[2 * kb + 1][3], hi[3], lo[3]);
                put_tile(out + Lay::M + (i * 4 + kb) * 1024, lane, hi, lo);
            }
        }
    }
    // e^(L_t) q as rows of tokens, e^(L_C - L_s) k transposed
    for (int tile = warp; tile < 4 * KS; tile += NT / 32) {
        const int i = tile / KS, ks = tile % KS;
        uint32_t h4[4], l4[4];
        int at = (i * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8;
        ldsm_x4(h4, smem_u32(Qh + at));
        ldsm_x4(l4, smem_u32(Ql + at));
#pragma unroll
        for (int r = 0; r < 4; ++r) {                  // registers 0, 2: token g8 of the sixteen; 1, 3: eight later
            const float f = eL[i * 16 + g8 + (r & 1) * 8];
            const float2 x = bf16_pair(h4[r]), y = bf16_pair(l4[r]);
            split2(f * (x.x + y.x), f * (x.y + y.y), h4[r], l4[r]);
        }
        put_tile(out + Lay::Q + tile * 1024, lane, h4, l4);
        // K^T: sixteen key components (ks) by sixteen tokens (i)
        at = (i * 16 + b4 * 8 + l7) * LDK + ks * 16 + b3 * 8;
        ldsm_x4_t(h4, smem_u32(Kh + at));
        ldsm_x4_t(l4, smem_u32(Kl + at));
#pragma unroll
        for (int r = 0; r < 4; ++r) {                  // registers 0, 1: tokens pc, pc + 1 of the sixteen; 2, 3: eight later
            const int t = i * 16 + pc + (r >> 1) * 8;
            const float f0 = expf(lend - L[t]), f1 = expf(lend - L[t + 1]);
            const float2 x = bf16_pair(h4[r]), y = bf16_pair(l4[r]);
            split2(f0 * (x.x + y.x), f1 * (x.y + y.y), h4[r], l4[r]);
        }
        put_tile(out + Lay::K + (ks * 4 + i) * 1024, lane, h4, l4);
    }
    if (threadIdx.x == 0) *reinterpret_cast<float*>(out + Lay::U0 + (long)C * P * 4) = expf(lend);
    __syncthreads();
    // forward substitution: a thread takes a column of the right sides, first those of W, then those of U0
    float* u0 = reinterpret_cast<float*>(out + Lay::U0);
    for (int base = 0; base < N + P; base += NT) {
        const int col = base + threadIdx.x;
        float x[C];
        if (col < N) {
#pragma unroll
            for (int t = 0; t < C; ++t) x[t] = bt[t] * eL[t] * (__bfloat162float(Kh[t * LDK + col]) + __bfloat162float(Kl[t * LDK + col]));
        } else {
            const bf16* vc = v + (long)t0 * ldv + (long)h * P + (col < N + P ? col - N : 0);
#pragma unroll
            for (int t = 0; t < C; ++t) x[t] = t < n ? bt[t] * __bfloat162float(vc[(long)t * ldv]) : 0.f;
        }
#pragma unroll
        for (int s = 0; s < C - 1; ++s) {
#pragma unroll
            for (int t4 = (s + 1) / 4 * 4; t4 < C; t4 += 4) {
                const float4 a = *reinterpret_cast<const float4*>(At + s * LDA + t4);       // (zero up to the diagonal)
                if (t4 > s) x[t4] = fmaf(-a.x, x[s], x[t4]);
                if (t4 + 1 > s) x[t4 + 1] = fmaf(-a.y, x[s], x[t4 + 1]);
                if (t4 + 2 > s) x[t4 + 2] = fmaf(-a.z, x[s], x[t4 + 2]);
                x[t4 + 3] = fmaf(-a.w, x[s], x[t4 + 3]);
            }
        }
        if (col >= N && col < N + P) {
#pragma unroll
            for (int t = 0; t < C; ++t) u0[t * P + col - N] = x[t];
        }
        if (base == 0) {
            // -W in two terms in the place of q (whose tiles are out), then to fragments
            if (col < NP) {
#pragma unroll
                for (int t = 0; t < C; ++t) {
                    const float y = col < N ? -x[t] : 0.f;
                    const bf16 hi = __float2bfloat16_rn(y);
                    Qh[t * LDK + col] = hi;
                    Ql[t * LDK + col] = __float2bfloat16_rn(y - __bfloat162float(hi));
                }
            }
            __syncthreads();
            for (int tile = warp; tile < 4 * KS; tile += NT / 32) {
                const int i = tile / KS, ks = tile % KS;
                const int at = (i * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8;
                uint32_t h4[4], l4[4];
                ldsm_x4(h4, smem_u32(Qh + at));
                ldsm_x4(l4, smem_u32(Ql + at));
                put_tile(out + Lay::W + tile * 1024, lane, h4, l4);
            }
        }
    }
}

struct Frag { uint4 hi, lo; };
__device__ __forceinline__ Frag get_tile(const uint8_t* tile, int lane) {
    const uint4* p = reinterpret_cast<const uint4*>(tile);
    return Frag{__ldcg(p + lane), __ldcg(p + 32 + lane)};
}
__device__ __forceinline__ void as_regs(const uint4& v, uint32_t (&r)[4]) { r[0] = v.x, r[1] = v.y, r[2] = v.z, r[3] = v.w; }

// acc[16 rows][32 columns] += (the fragment's sixteen rows and sixteen k) times the 16 x 32 block of X (two terms, rows LDS_)
__device__ __forceinline__ void times_block(float (&acc)[4][4], const Frag& f, const bf16* Xh, const bf16* Xl, int row, int lane) {
    const int l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    uint32_t ah[4], al[4], xh[2][4], xl[2][4];
    as_regs(f.hi, ah), as_regs(f.lo, al);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int at = (row + l7 + b3 * 8) * LDS_ + j * 16 + b4 * 8;
        ldsm_x4_t(xh[j], smem_u32(Xh + at));
        ldsm_x4_t(xl[j], smem_u32(Xl + at));
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        mma_bf16(acc[2 * j], ah, xh[j][0], xh[j][1]);
        mma_bf16(acc[2 * j + 1], ah, xh[j][2], xh[j][3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        mma_bf16(acc[2 * j], al, xh[j][0], xh[j][1]);
        mma_bf16(acc[2 * j + 1], al, xh[j][2], xh[j][3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        mma_bf16(acc[2 * j], ah, xl[j][0], xl[j][1]);
        mma_bf16(acc[2 * j + 1], ah, xl[j][2], xl[j][3]);
    }
}

// grid: (sequence, head, PT columns of the state).  Warps 0..3 make U (sixteen tokens each), warps 4..7 O; warp w also keeps
// rows 16 w .. 16 w + 15 of the state (as far as there are that many).
template <int NP>
__global__ void __launch_bounds__(NT, 1)
delta_head_walk_kernel(const uint8_t* ws, float* __restrict__ state, long state_stride, float* __restrict__ y, const int* seq_start,
                       const int* seq_slot, int H, int N, int P) {
    constexpr int KS = NP / 16;
    using Lay = Layout<NP>;
    __shared__ __align__(16) bf16 Sh[NP * LDS_], Sl[NP * LDS_], Uh[C * LDS_], Ul[C * LDS_];
    pdl_launch_dependents();
    const int ptiles = (P + PT - 1) / PT;
    int bid = blockIdx.x;
    const int p0 = (bid % ptiles) * PT;
    bid /= ptiles;
    const int h = bid % H, b = bid / H;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, pc = (lane & 3) * 2;
    const bool makes_u = warp < 4, keeps = warp < KS;
    const int i = warp & 3;
    pdl_wait();
    const int s0 = seq_start[b], s1 = seq_start[b + 1];
    if (s1 <= s0) return;
    float* st = state + (long)seq_slot[b] * state_stride + (long)h * N * P;
    const long per = Lay::bytes(P);
    const uint8_t* src = ws + ((long)(s0 / C + b) * H + h) * per;
    float S[4][4];
    auto each = [&](auto&& f) {                        // this warp's piece of the state: f(row, column, j, first register)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) f(warp * 16 + g8 + hi * 8, j * 8 + pc, j, 2 * hi);
    };
    auto share = [&]() {                               // to shared memory in two terms
        each([&](int r, int c, int j, int e) {
            split2(S[j][e], S[j][e + 1], *reinterpret_cast<uint32_t*>(Sh + r * LDS_ + c), *reinterpret_cast<uint32_t*>(Sl + r * LDS_ + c));
        });
    };
    Frag wq[KS];                                       // rows of -W (warps 0..3) or of e^L q
    float u0[4][4];
    auto ahead = [&](const uint8_t* from) {            // what the first phase of a chunk takes
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) wq[ks] = get_tile(from + (makes_u ? Lay::W : Lay::Q) + (i * KS + ks) * 1024, lane);
        const float* u = reinterpret_cast<const float*>(from + Lay::U0);
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                float2 x = make_float2(0.f, 0.f);
                const int p = p0 + j * 8 + pc;
                if (makes_u && p < P) x = __ldcg(reinterpret_cast<const float2*>(u + (long)(i * 16 + g8 + hi * 8) * P + p));
                u0[j][2 * hi] = x.x, u0[j][2 * hi + 1] = x.y;
            }
    };
    ahead(src);
    if (keeps) {
        each([&](int r, int c, int j, int e) {
            float2 x = make_float2(0.f, 0.f);
            if (r < N && p0 + c < P) x = *reinterpret_cast<const float2*>(st + (long)r * P + p0 + c);
            S[j][e] = x.x, S[j][e + 1] = x.y;
        });
        share();
    }
    __syncthreads();
    for (int base = s0; base < s1; base += C, src += (long)H * per) {
        const int n = min(C, s1 - base);
        Frag kt[4], m[4];
        float fade = 0.f;
        if (keeps) {
#pragma unroll
            for (int s = 0; s < 4; ++s) kt[s] = get_tile(src + Lay::K + (warp * 4 + s) * 1024, lane);
            fade = __ldcg(reinterpret_cast<const float*>(src + Lay::U0 + (long)C * P * 4));
        }
        if (!makes_u) {
#pragma unroll
            for (int s = 0; s < 4; ++s)
                if (s <= i) m[s] = get_tile(src + Lay::M + (i * 4 + s) * 1024, lane);
        }
        float acc[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[j][e] = u0[j][e];
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) times_block(acc, wq[ks], Sh, Sl, ks * 16, lane);
        if (makes_u) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    const int at = (i * 16 + g8 + hi * 8) * LDS_ + j * 8 + pc;
                    split2(acc[j][2 * hi], acc[j][2 * hi + 1], *reinterpret_cast<uint32_t*>(Uh + at), *reinterpret_cast<uint32_t*>(Ul + at));
                }
        }
        __syncthreads();                               // U is there, the state in shared memory has been read
        if (base + C < s1) ahead(src + (long)H * per);
        if (keeps) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] *= fade;
#pragma unroll
            for (int s = 0; s < 4; ++s) times_block(S, kt[s], Uh, Ul, s * 16, lane);
            share();
        }
        if (!makes_u) {
#pragma unroll
            for (int s = 0; s < 4; ++s)
                if (s <= i) times_block(acc, m[s], Uh, Ul, s * 16, lane);
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                const int t = i * 16 + g8 + hi * 8;
                if (t >= n) continue;
                float* yr = y + (long)(base + t) * H * P + (long)h * P + p0 + pc;
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (p0 + j * 8 < P) *reinterpret_cast<float2*>(yr + j * 8) = make_float2(acc[j][2 * hi], acc[j][2 * hi + 1]);
            }
        }
        __syncthreads();                               // the new state is there, U has been read
    }
    if (keeps)
        each([&](int r, int c, int j, int e) {
            if (r < N && p0 + c < P) *reinterpret_cast<float2*>(st + (long)r * P + p0 + c) = make_float2(S[j][e], S[j][e + 1]);
        });
}

template <int NP>
int launch(const float* qn, const float* kn, const float* dec, const float* beta, const bf16* v, long ldv, float* state,
           long state_stride, float* y, uint8_t* ws, const int* seq_start, const int* seq_slot, int n_seqs, int max_new, int H, int N,
           int P, int heads_per_group, cudaStream_t stream) {
    static bool configured = false;
    constexpr size_t smem = prep_smem<NP>();
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(delta_head_prep_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const dim3 pgrid((unsigned)((max_new + C - 1) / C), (unsigned)n_seqs, (unsigned)H);
    cudaError_t e = launch_pdl(delta_head_prep_kernel<NP>, pgrid, dim3(NT), smem, stream, qn, kn, dec, beta, v, ldv, ws, seq_start, H, N,
                               P, heads_per_group);
    if (e != cudaSuccess) return (int)e;
    const unsigned grid = (unsigned)((long)n_seqs * H * ((P + PT - 1) / PT));
    return plm_status_of(launch_pdl(delta_head_walk_kernel<NP>, dim3(grid), dim3(NT), 0, stream, ws, state, state_stride, y, seq_start,
                                    seq_slot, H, N, P));
}

}  // namespace

// Bytes of workspace per (chunk of 64 tokens, head); a sequence's chunks start at number seq_start / 64 + sequence.
extern "C" int plm_delta_head_chunk_bytes(int N, int P) {
    return (int)(N <= 32 ? Layout<32>::bytes(P) : N <= 64 ? Layout<64>::bytes(P) : Layout<128>::bytes(P));
}

// qn, kn [T, G * N], dec (logarithms), beta [T, H] fp32 as plm_delta_prep leaves them with one decay a head; v [T, H * P] bf16
// (N a multiple of 16 up to 128, P of 8); state [slots][>= H * N * P] fp32; y [T, H * P] fp32; ws 16-byte aligned,
// (n_tokens / 64 + n_seqs + 1) * H * plm_delta_head_chunk_bytes(N, P) bytes.
extern "C" int plm_delta_head_chunk_scan(const float* qn, const float* kn, const float* dec, const float* beta, const void* v, long ldv,
                                         float* state, long state_stride, float* y, void* ws, const int* seq_start,
                                         const int* seq_slot, int n_seqs, int max_new, int H, int N, int P, int heads_per_group,
                                         cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return PLM_OK;
    if (H <= 0 || H > 65535 || n_seqs > 65535 || N <= 0 || N % 16 || N > 128 || P <= 0 || P % 8 || heads_per_group <= 0 || H % heads_per_group)
        return PLM_ERR_SHAPE;
    if ((((uintptr_t)qn | (uintptr_t)kn | (uintptr_t)ws | (uintptr_t)y | (uintptr_t)state) & 15) || state_stride % 2) return PLM_ERR_ALIGN;
#define DH(NP_)                                                                                                                  \
    return launch<NP_>(qn, kn, dec, beta, (const bf16*)v, ldv, state, state_stride, y, (uint8_t*)ws, seq_start, seq_slot, n_seqs, \
                       max_new, H, N, P, heads_per_group, stream)
    if (N <= 32) DH(32);
    if (N <= 64) DH(64);
    DH(128);
#undef DH
}
