// Linear attention with one constant decay a head, for prompts, in bfloat16 on the tensor cores (mma.sync m16n8k16, fp32
// accumulation): the recurrence
//   S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// taken 64 tokens at a time.  With S the state before a chunk of n tokens, t and s counting inside it:
//   o_t = d^(t+1) S^T q_t + sum_{s <= t} d^(t-s) (q_t . k_s) v_s
//   S  <- d^n S + sum_s k_s (d^(n-1-s) v_s)^T
// Every exponent is >= 0 and the powers come from a table [heads][65] (float32, made from the decay in double precision),
// so nothing over- or underflows however strong the decay.
//
// q, k and v are the rows of the projections or their activations SiLU(row), rounded to bf16 as activations are elsewhere.
// What the products take that is not such an activation (the chunk's weights d^(t-s) q.k, the state where it is read, the
// decayed keys) goes in as two bf16 terms, x = hi + lo with hi = bf16(x) and lo = bf16(x - hi), so that it keeps 16
// bits; the state itself is fp32 in registers from chunk to chunk and in the cache.
//
// ROT: queries and keys are rotated by their positions on the way in (pairs (i, i + half) of a head, angles from a table of
// fp32 cosines and sines) and the keys multiplied by a constant.  Both happen in fp32, so the results are not activations
// that a bf16 run rounds: they go into the products as two terms too (hi hi + hi lo + lo hi).
//
// One block per (sequence, head, 128 value columns, segment), 8 warps.  For o a warp has 16 of the chunk's tokens and half
// of the columns, for the state 16 of its rows.  A chunk's rows arrive through cp.async while the chunk before is worked
// on.  Long prompts are cut into segments that run side by side, in three passes as in recurrent.cu: each segment's own
// contribution from zero (LOCAL), the state at every segment's start (decay_combine_kernel), and the walk that writes o
// (FINAL; WHOLE where there is one segment).
//
// Steps of single tokens take decay_step_kernel, which streams the state through once.
#include "mma_common.cuh"

namespace {

constexpr int NT = 256, C = 64, PT = 128;
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
    const float *cos_t, *sin_t;                        // ROT: [positions][half]
    const int* tok_pos;
    int half;                                          // rotated pairs of a head (0: none)
    float k_scale;
    float* seg_state;                                  // [seq][segment][H][N][P]
};

__device__ __forceinline__ float silu_f(float x) { return __fdividef(x, 1.f + __expf(-x)); }      // (rounded to bf16 right away)

// eight activations of a row: SiLU where asked for, rounded to bf16
__device__ __forceinline__ uint4 act8(uint4 raw, bool silu) {
    if (!silu) return raw;
    uint32_t* w = reinterpret_cast<uint32_t*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(w + i);
        w[i] = bf16_bits(__floats2bfloat162_rn(silu_f(__low2float(h)), silu_f(__high2float(h))));
    }
    return raw;
}

template <int NP, bool ROT> constexpr size_t smem_bytes() {
    // q and k (rotated: in two terms), v; the state in two terms; rows as they arrive; the powers
    return (size_t)((ROT ? 4 : 2) * C * (NP + 8) + C * LDV + 2 * NP * LDV + C * (2 * NP + PT)) * sizeof(bf16) + (POW_N + 3) / 4 * 4 * sizeof(float);
}

// Eight pairs (u, v) of a row turned by their angles (turn: whether there are any), times `scale`, as two bf16 terms each.
__device__ __forceinline__ void turn8(const bf16* row, int cu, int cv, bool turn, const float4 (&cs)[4], float scale, bf16* hi, bf16* lo) {
    const uint4 u = *reinterpret_cast<const uint4*>(row + cu), v = *reinterpret_cast<const uint4*>(row + cv);
    const uint32_t *uw = reinterpret_cast<const uint32_t*>(&u), *vw = reinterpret_cast<const uint32_t*>(&v);
    const float *c = reinterpret_cast<const float*>(cs), *sn = c + 8;
    uint32_t uh[4], ul[4], vh[4], vl[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 x = bf16_pair(uw[i]), y = bf16_pair(vw[i]);
        float2 p = x, q = y;
        if (turn) {
            p = make_float2(rope_first(x.x, y.x, c[2 * i], sn[2 * i]), rope_first(x.y, y.y, c[2 * i + 1], sn[2 * i + 1]));
            q = make_float2(rope_second(x.x, y.x, c[2 * i], sn[2 * i]), rope_second(x.y, y.y, c[2 * i + 1], sn[2 * i + 1]));
        }
        split2(p.x * scale, p.y * scale, uh[i], ul[i]);
        split2(q.x * scale, q.y * scale, vh[i], vl[i]);
    }
    *reinterpret_cast<uint4*>(hi + cu) = make_uint4(uh[0], uh[1], uh[2], uh[3]);
    *reinterpret_cast<uint4*>(lo + cu) = make_uint4(ul[0], ul[1], ul[2], ul[3]);
    *reinterpret_cast<uint4*>(hi + cv) = make_uint4(vh[0], vh[1], vh[2], vh[3]);
    *reinterpret_cast<uint4*>(lo + cv) = make_uint4(vl[0], vl[1], vl[2], vl[3]);
}

// One pair, for rotations whose pairs do not come in eights.
__device__ __forceinline__ void turn1(const bf16* row, int cu, int cv, bool turn, float c, float sn, float scale, bf16* hi, bf16* lo) {
    const float x = __bfloat162float(row[cu]), y = __bfloat162float(row[cv]);
    const float p = (turn ? rope_first(x, y, c, sn) : x) * scale, q = (turn ? rope_second(x, y, c, sn) : y) * scale;
    hi[cu] = __float2bfloat16_rn(p);
    hi[cv] = __float2bfloat16_rn(q);
    lo[cu] = __float2bfloat16_rn(p - __bfloat162float(hi[cu]));
    lo[cv] = __float2bfloat16_rn(q - __bfloat162float(hi[cv]));
}

template <int NP, int PASS, bool ROT>
__global__ void __launch_bounds__(NT, 1) decay_chunk_kernel(const Args a) {
    constexpr int LDK = NP + 8, KS = NP / 16;
    constexpr int PG = NP / 16, TURNS = C * PG / NT;   // groups of eight pairs in a row; groups a thread turns
    constexpr int ROW_GROUPS = NP / 16, COL_GROUPS = 8 / ROW_GROUPS, SJ = PT / COL_GROUPS / 8;    // a warp's share of the state
    constexpr int OJ = PT / 2 / 8;                     // a warp's column tiles of o
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);      // [C][LDK]
    bf16* Ks = Qs + C * LDK;                           // [C][LDK]
    bf16* Qlo = Ks + C * LDK;                          // ROT: the second terms of q and k
    bf16* Klo = Qlo + (ROT ? C * LDK : 0);
    bf16* Vs = Klo + (ROT ? C * LDK : 0);              // [C][LDV]: v
    bf16* Shi = Vs + C * LDV;                          // [NP][LDV]: the state in two terms
    bf16* Slo = Shi + NP * LDV;
    bf16* Rq = Slo + NP * LDV;                         // rows as they arrive: q [C][NP], k [C][NP], v [C][PT]
    bf16* Rk = Rq + C * NP;
    bf16* Rv = Rk + C * NP;
    float* pw = reinterpret_cast<float*>(Rv + C * PT); // [65]
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

    auto request = [&](int base) {                     // the rows of the chunk that starts at token `base`
        const int n = min(C, t1 - base);
#pragma unroll
        for (int idx = threadIdx.x; idx < C * (NP / 8); idx += NT) {
            const int r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
            const bool in = r < n && c < N;
            const long row = in ? base + r : base;
            const int col = in ? c : 0;
            cp_async16(smem_u32(Rk + r * NP + c), a.k + row * a.ldk + (long)h * N + col, in);
            if (PASS != PASS_LOCAL) cp_async16(smem_u32(Rq + r * NP + c), a.q + row * a.ldq + (long)h * N + col, in);
        }
#pragma unroll
        for (int idx = threadIdx.x; idx < C * (PT / 8); idx += NT) {
            const int r = idx / (PT / 8), c = (idx % (PT / 8)) * 8;
            const bool in = r < n && p0 + c < P;
            cp_async16(smem_u32(Rv + r * PT + c), a.v + (long)(in ? base + r : base) * a.ldv + (long)h * P + (in ? p0 + c : p0), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request(t0);

    // this warp's piece of the state: rows sr + lane / 4 (+ 8), columns p0 + sc + 8 j + 2 (lane % 4) (+ 1)
    const int sr = (warp % ROW_GROUPS) * 16, sc = (warp / ROW_GROUPS) * (PT / COL_GROUPS);
    const int pc = (lane & 3) * 2;
    float S[SJ][4];
#pragma unroll
    for (int j = 0; j < SJ; ++j)
#pragma unroll
        for (int hi = 0; hi < 2; ++hi) {
            const int n = sr + (lane >> 2) + hi * 8, p = p0 + sc + j * 8 + pc;
            float2 x = make_float2(0.f, 0.f);
            if (init && n < N && p < P) x = *reinterpret_cast<const float2*>(init + (long)n * P + p);
            S[j][2 * hi] = x.x;
            S[j][2 * hi + 1] = x.y;
        }

    // this warp's piece of o: tokens 16 tg .. 16 tg + 15 of the chunk, columns oc .. oc + 63 (later tokens meet more keys:
    // the two warps of a scheduler take a late and an early group)
    const int tg = warp < 4 ? warp : 7 - warp, oc = (warp >> 2) * (PT / 2);
    const bool silu = a.silu;
    const int l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    const int half = ROT ? a.half : 0;
    const int pos0 = ROT && half > 0 ? a.tok_pos[t0] : 0;
    const bool by8 = half % 8 == 0;
    for (int base = t0; base < t1; base += C) {
        const int n = min(C, t1 - base);               // tokens of this chunk
        float4 cs[TURNS][4];                           // the angles of this thread's groups: asked for before the wait
        if (ROT && by8) {
#pragma unroll
            for (int i = 0; i < TURNS; ++i) {
                const int idx = threadIdx.x + i * NT, r = idx / PG, g8 = (idx % PG) * 8;
                if (g8 < half && r < n) {
                    const long at = (long)(pos0 + base - t0 + r) * half + g8;
                    const float4 *cp = reinterpret_cast<const float4*>(a.cos_t + at), *sp = reinterpret_cast<const float4*>(a.sin_t + at);
                    cs[i][0] = cp[0], cs[i][1] = cp[1], cs[i][2] = sp[0], cs[i][3] = sp[1];
                } else {
                    cs[i][0] = cs[i][1] = cs[i][2] = cs[i][3] = make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                               // this chunk's rows are there, the chunk before has been read
        if (ROT && by8) {
#pragma unroll
            for (int i = 0; i < TURNS; ++i) {
                const int idx = threadIdx.x + i * NT, r = idx / PG, g = idx % PG;
                const bool turn = g * 8 < half;
                const int cu = turn ? g * 8 : 2 * half + (g - half / 8) * 16, cv = turn ? half + g * 8 : cu + 8;
                if (PASS != PASS_LOCAL) turn8(Rq + r * NP, cu, cv, turn, cs[i], 1.f, Qs + r * LDK, Qlo + r * LDK);
                turn8(Rk + r * NP, cu, cv, turn, cs[i], a.k_scale, Ks + r * LDK, Klo + r * LDK);
            }
        } else if (ROT) {
            for (int idx = threadIdx.x; idx < C * (NP / 2); idx += NT) {
                const int r = idx / (NP / 2), g = idx % (NP / 2);
                const bool turn = g < half;
                const int cu = turn ? g : 2 * half + (g - half) * 2, cv = turn ? half + g : cu + 1;
                const long at = (long)(pos0 + base - t0 + min(r, n - 1)) * half + (turn ? g : 0);
                const float c = a.cos_t[at], sn = a.sin_t[at];
                if (PASS != PASS_LOCAL) turn1(Rq + r * NP, cu, cv, turn, c, sn, 1.f, Qs + r * LDK, Qlo + r * LDK);
                turn1(Rk + r * NP, cu, cv, turn, c, sn, a.k_scale, Ks + r * LDK, Klo + r * LDK);
            }
        } else {
#pragma unroll
            for (int idx = threadIdx.x; idx < C * (NP / 8); idx += NT) {
                const int r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
                if (PASS != PASS_LOCAL) *reinterpret_cast<uint4*>(Qs + r * LDK + c) = act8(*reinterpret_cast<const uint4*>(Rq + r * NP + c), silu);
                *reinterpret_cast<uint4*>(Ks + r * LDK + c) = act8(*reinterpret_cast<const uint4*>(Rk + r * NP + c), silu);
            }
        }
#pragma unroll
        for (int idx = threadIdx.x; idx < C * (PT / 8); idx += NT) {
            const int r = idx / (PT / 8), c = (idx % (PT / 8)) * 8;
            *reinterpret_cast<uint4*>(Vs + r * LDV + c) = act8(*reinterpret_cast<const uint4*>(Rv + r * PT + c), silu);
        }
        if (PASS != PASS_LOCAL) {
#pragma unroll
            for (int j = 0; j < SJ; ++j)
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    uint32_t xh, xl;
                    split2(S[j][2 * hi], S[j][2 * hi + 1], xh, xl);
                    const int at = (sr + (lane >> 2) + hi * 8) * LDV + sc + j * 8 + pc;
                    *reinterpret_cast<uint32_t*>(Shi + at) = xh;
                    *reinterpret_cast<uint32_t*>(Slo + at) = xl;
                }
        }
        __syncthreads();
        if (base + C < t1) request(base + C);
        if (PASS != PASS_LOCAL && tg * 16 < n && p0 + oc < P) {
            const int tl = tg * 16 + (lane >> 2);      // this lane's first token; the other is tl + 8
            uint32_t qa[KS][4];
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) ldsm_x4(qa[ks], smem_u32(Qs + (tg * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8));
            float o[OJ][4];
#pragma unroll
            for (int j = 0; j < OJ; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {          // S^T q: what comes from the chunks before
                uint32_t ql[4];
                if (ROT) ldsm_x4(ql, smem_u32(Qlo + (tg * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8));
#pragma unroll
                for (int term = 0; term < 2; ++term) {
                    const bf16* Sx = term ? Slo : Shi;
                    uint32_t f[OJ / 2][4];
#pragma unroll
                    for (int j = 0; j < OJ / 2; ++j)
                        ldsm_x4_t(f[j], smem_u32(Sx + (ks * 16 + l7 + b3 * 8) * LDV + oc + j * 16 + b4 * 8));
#pragma unroll
                    for (int j = 0; j < OJ / 2; ++j) {
                        mma_bf16(o[2 * j], qa[ks], f[j][0], f[j][1]);
                        mma_bf16(o[2 * j + 1], qa[ks], f[j][2], f[j][3]);
                    }
                    if (ROT && term == 0) {
#pragma unroll
                        for (int j = 0; j < OJ / 2; ++j) {
                            mma_bf16(o[2 * j], ql, f[j][0], f[j][1]);
                            mma_bf16(o[2 * j + 1], ql, f[j][2], f[j][3]);
                        }
                    }
                }
            }
            const float dlo = pw[tl + 1], dhi = pw[tl + 9];
#pragma unroll
            for (int j = 0; j < OJ; ++j) {
                o[j][0] *= dlo; o[j][1] *= dlo;
                o[j][2] *= dhi; o[j][3] *= dhi;
            }
#pragma unroll 1
            for (int kb = 0; kb <= tg; ++kb) {         // the chunk's own keys, 16 at a time
                float w[2][2][4];                      // two sums a tile: even and odd steps of the key size
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) w[0][i][e] = w[1][i][e] = 0.f;
#pragma unroll
                for (int ks = 0; ks < KS; ++ks) {
                    uint32_t kf[4];
                    ldsm_x4(kf, smem_u32(Ks + (kb * 16 + l7 + b4 * 8) * LDK + ks * 16 + b3 * 8));
                    mma_bf16(w[ks & 1][0], qa[ks], kf[0], kf[1]);
                    mma_bf16(w[ks & 1][1], qa[ks], kf[2], kf[3]);
                    if (ROT) {
                        uint32_t ql[4], kl[4];
                        ldsm_x4(ql, smem_u32(Qlo + (tg * 16 + (lane & 15)) * LDK + ks * 16 + b4 * 8));
                        ldsm_x4(kl, smem_u32(Klo + (kb * 16 + l7 + b4 * 8) * LDK + ks * 16 + b3 * 8));
                        mma_bf16(w[ks & 1][0], ql, kf[0], kf[1]);
                        mma_bf16(w[ks & 1][1], ql, kf[2], kf[3]);
                        mma_bf16(w[ks & 1][0], qa[ks], kl[0], kl[1]);
                        mma_bf16(w[ks & 1][1], qa[ks], kl[2], kl[3]);
                    }
                }
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int dist = tl + (e >> 1) * 8 - (kb * 16 + i * 8 + pc + (e & 1));
                        w[0][i][e] = dist >= 0 ? (w[0][i][e] + w[1][i][e]) * pw[dist] : 0.f;
                    }
                uint32_t ah[4], al[4];
                split2(w[0][0][0], w[0][0][1], ah[0], al[0]);
                split2(w[0][0][2], w[0][0][3], ah[1], al[1]);
                split2(w[0][1][0], w[0][1][1], ah[2], al[2]);
                split2(w[0][1][2], w[0][1][3], ah[3], al[3]);
                uint32_t vf[OJ / 2][4];
#pragma unroll
                for (int j = 0; j < OJ / 2; ++j)
                    ldsm_x4_t(vf[j], smem_u32(Vs + (kb * 16 + l7 + b3 * 8) * LDV + oc + j * 16 + b4 * 8));
#pragma unroll
                for (int j = 0; j < OJ / 2; ++j) {
                    mma_bf16(o[2 * j], ah, vf[j][0], vf[j][1]);
                    mma_bf16(o[2 * j + 1], ah, vf[j][2], vf[j][3]);
                }
#pragma unroll
                for (int j = 0; j < OJ / 2; ++j) {
                    mma_bf16(o[2 * j], al, vf[j][0], vf[j][1]);
                    mma_bf16(o[2 * j + 1], al, vf[j][2], vf[j][3]);
                }
            }
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                const int t = tl + hi * 8;
                if (t >= n) continue;
                float* yr = a.y + (long)(base + t) * a.ldy + (long)h * P + p0 + oc + pc;
#pragma unroll
                for (int j = 0; j < OJ; ++j)
                    if (p0 + oc + j * 8 < P) *reinterpret_cast<float2*>(yr + j * 8) = make_float2(o[j][2 * hi], o[j][2 * hi + 1]);
            }
        }
        // the state: d^n S + (decayed K)^T V, token s of the chunk's keys times d^(n-1-s) in registers
        const float dn = pw[n];
#pragma unroll
        for (int j = 0; j < SJ; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[j][e] *= dn;
        if (p0 + sc < P) {
#pragma unroll
            for (int sb = 0; sb < C / 16; ++sb) {
                if (sb * 16 >= n) break;
                const uint32_t at = smem_u32(Ks + (sb * 16 + b4 * 8 + l7) * LDK + sr + b3 * 8);
                uint32_t ka[4], kl[4], ah[4], al[4];
                ldsm_x4_t(ka, at);
                if (ROT) ldsm_x4_t(kl, at + (uint32_t)((Klo - Ks) * sizeof(bf16)));
#pragma unroll
                for (int i = 0; i < 4; ++i) {          // registers 0, 1: tokens pc, pc + 1 of the sixteen; 2, 3: eight later
                    const int tok = sb * 16 + pc + (i >> 1) * 8;
                    const float g0 = tok < n ? pw[n - 1 - tok] : 0.f, g1 = tok + 1 < n ? pw[n - 2 - tok] : 0.f;
                    float2 x = bf16_pair(ka[i]);
                    if (ROT) {
                        const float2 y = bf16_pair(kl[i]);
                        x = make_float2(x.x + y.x, x.y + y.y);
                    }
                    split2(g0 * x.x, g1 * x.y, ah[i], al[i]);
                }
#pragma unroll
                for (int j = 0; j < SJ / 2; ++j) {
                    uint32_t f[4];
                    ldsm_x4_t(f, smem_u32(Vs + (sb * 16 + l7 + b3 * 8) * LDV + sc + j * 16 + b4 * 8));
                    mma_bf16(S[2 * j], ah, f[0], f[1]);
                    mma_bf16(S[2 * j + 1], ah, f[2], f[3]);
                    mma_bf16(S[2 * j], al, f[0], f[1]);
                    mma_bf16(S[2 * j + 1], al, f[2], f[3]);
                }
            }
        }
    }
    float* dst = PASS == PASS_LOCAL ? sg : (PASS == PASS_WHOLE || seg == n_segs - 1) ? st : nullptr;
    if (dst) {
#pragma unroll
        for (int j = 0; j < SJ; ++j)
#pragma unroll
            for (int hi = 0; hi < 2; ++hi) {
                const int n = sr + (lane >> 2) + hi * 8, p = p0 + sc + j * 8 + pc;
                if (n < N && p < P) *reinterpret_cast<float2*>(dst + (long)n * P + p) = make_float2(S[j][2 * hi], S[j][2 * hi + 1]);
            }
    }
}

// One token for each sequence: S <- d S + k v^T and o = S^T q in one pass over the state.  A block per (64 value columns,
// head, sequence); 16 threads hold four columns each of a row, 16 rows at a time; the rows' shares of o are added in
// the order of the 16 row groups.  q, k and v are fp32 here, their activations rounded to the run's type; with a rotation
// (half > 0 pairs (i, i + half), angles of position tok_pos[b]) and a factor on the keys, both in fp32 and kept so.
constexpr int STEP_NT = 256, STEP_COLS = 64;
template <typename T>
__global__ void __launch_bounds__(STEP_NT)
decay_step_kernel(const T* q, const T* k, const T* v, long ldq, long ldk, long ldv,
                  const float* decay, float* __restrict__ state, long state_stride, float* __restrict__ y, long ldy,
                  const int* seq_slot, int N, int P, int silu, const float* cos_t, const float* sin_t, const int* tok_pos,
                  int half, float k_scale) {
    extern __shared__ float step_sm[];                 // q [N], k [N], shares [16][64]
    float* qs = step_sm;
    float* ks = qs + N;
    float4* share = reinterpret_cast<float4*>(step_sm + (2 * N + 3) / 4 * 4);
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.z, h = blockIdx.y;
    auto act = [&](float x) { return silu ? to_f32<T>(from_f32<T>(x / (1.f + expf(-x)))) : x; };
    const T *qr = q + b * ldq + (long)h * N, *kr = k + b * ldk + (long)h * N;
    if (half > 0) {
        const long at = (long)tok_pos[b] * half;
        for (int i = threadIdx.x; i < half; i += STEP_NT) {
            const float c = cos_t[at + i], sn = sin_t[at + i];
            const float q0 = to_f32<T>(qr[i]), q1 = to_f32<T>(qr[i + half]), k0 = to_f32<T>(kr[i]), k1 = to_f32<T>(kr[i + half]);
            qs[i] = rope_first(q0, q1, c, sn), qs[i + half] = rope_second(q0, q1, c, sn);
            ks[i] = rope_first(k0, k1, c, sn) * k_scale, ks[i + half] = rope_second(k0, k1, c, sn) * k_scale;
        }
    }
    for (int i = 2 * half + threadIdx.x; i < N; i += STEP_NT) {
        qs[i] = act(to_f32<T>(qr[i]));
        ks[i] = act(to_f32<T>(kr[i])) * k_scale;
    }
    const int cq = threadIdx.x & 15, rg = threadIdx.x >> 4;
    const int p = blockIdx.x * STEP_COLS + cq * 4;
    const float d = decay[h];
    float4 vv = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool in = p < P;                             // P is a multiple of 4
    if (in) {
        const T* vr = v + b * ldv + (long)h * P + p;
        vv = make_float4(act(to_f32<T>(vr[0])), act(to_f32<T>(vr[1])), act(to_f32<T>(vr[2])), act(to_f32<T>(vr[3])));
    }
    __syncthreads();
    float* st = state + (long)seq_slot[b] * state_stride + (long)h * N * P + p;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (in) {
        for (int n0 = rg; n0 < N; n0 += 128) {         // eight rows' values are asked for at once
            float4 x[8];
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (n0 + 16 * i < N) x[i] = *reinterpret_cast<const float4*>(st + (long)(n0 + 16 * i) * P);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int n = n0 + 16 * i;
                if (n >= N) break;
                const float kn = ks[n], qn = qs[n];
                x[i] = make_float4(fmaf(d, x[i].x, kn * vv.x), fmaf(d, x[i].y, kn * vv.y), fmaf(d, x[i].z, kn * vv.z), fmaf(d, x[i].w, kn * vv.w));
                *reinterpret_cast<float4*>(st + (long)n * P) = x[i];
                acc = make_float4(fmaf(x[i].x, qn, acc.x), fmaf(x[i].y, qn, acc.y), fmaf(x[i].z, qn, acc.z), fmaf(x[i].w, qn, acc.w));
            }
        }
    }
    share[rg * 16 + cq] = acc;
    __syncthreads();
    if (threadIdx.x < STEP_COLS) {
        const int c = threadIdx.x, pp = blockIdx.x * STEP_COLS + c;
        const float* sh = reinterpret_cast<const float*>(share) + c;
        float sum = sh[0];
#pragma unroll
        for (int r = 1; r < 16; ++r) sum += sh[r * STEP_COLS];
        if (pp < P) y[b * ldy + (long)h * P + pp] = sum;
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

// Rows for the walk token by token: q and k rotated and k scaled, as fp32 [T, 2 H N] (q's columns, then k's), and v as fp32
// [T, H P] where it is asked for.  One block per token.
template <typename T>
__global__ void rotate_rows_kernel(const T* q, const T* k, const T* v, long ldq, long ldk, long ldv, const float* cos_t,
                                   const float* sin_t, const int* tok_pos, int half, float k_scale, float* __restrict__ qk,
                                   float* __restrict__ vo, int H, int N, int P) {
    pdl_launch_dependents();
    pdl_wait();
    const long t = blockIdx.x;
    const T *qr = q + t * ldq, *kr = k + t * ldk;
    float *qo = qk + t * 2 * H * N, *ko = qo + (long)H * N;
    const long at = half > 0 ? (long)tok_pos[t] * half : 0;
    const int per = N - half;                          // a head's work items: its pairs, then what passes
    for (int idx = threadIdx.x; idx < H * per; idx += blockDim.x) {
        const int h = idx / per, i = idx % per, c0 = h * N + i;
        if (i < half) {
            const float c = cos_t[at + i], sn = sin_t[at + i];
            const float q0 = to_f32<T>(qr[c0]), q1 = to_f32<T>(qr[c0 + half]), k0 = to_f32<T>(kr[c0]), k1 = to_f32<T>(kr[c0 + half]);
            qo[c0] = rope_first(q0, q1, c, sn), qo[c0 + half] = rope_second(q0, q1, c, sn);
            ko[c0] = rope_first(k0, k1, c, sn) * k_scale, ko[c0 + half] = rope_second(k0, k1, c, sn) * k_scale;
        } else {
            qo[c0 + half] = to_f32<T>(qr[c0 + half]);
            ko[c0 + half] = to_f32<T>(kr[c0 + half]) * k_scale;
        }
    }
    if (vo)
        for (int i = threadIdx.x; i < H * P; i += blockDim.x) vo[t * H * P + i] = to_f32<T>(v[t * ldv + i]);
}

template <int NP, bool ROT>
int launch(const Args& a, cudaStream_t stream) {
    static bool configured = false;
    constexpr size_t smem = smem_bytes<NP, ROT>();
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_WHOLE, ROT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_LOCAL, ROT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_kernel<NP, PASS_FINAL, ROT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const unsigned blocks = (unsigned)((long)a.n_seqs * a.H * ((a.P + PT - 1) / PT));
    if (a.max_segs <= 1) return plm_status_of(launch_pdl(decay_chunk_kernel<NP, PASS_WHOLE, ROT>, dim3(blocks), dim3(NT), smem, stream, a));
    cudaError_t e = launch_pdl(decay_chunk_kernel<NP, PASS_LOCAL, ROT>, dim3(blocks, a.max_segs - 1), dim3(NT), smem, stream, a);
    if (e != cudaSuccess) return (int)e;
    const long quads = (long)a.n_seqs * a.H * a.N * a.P / 4;
    e = launch_pdl(decay_combine_kernel, dim3((unsigned)((quads + 127) / 128)), dim3(128), 0, stream, a);
    if (e != cudaSuccess) return (int)e;
    return plm_status_of(launch_pdl(decay_chunk_kernel<NP, PASS_FINAL, ROT>, dim3(blocks, a.max_segs), dim3(NT), smem, stream, a));
}

}  // namespace

// How a step of `n_tokens` tokens whose longest sequence brings `max_new` of them is cut: out[0] tokens per segment (a
// multiple of 64), out[1] segments of the longest sequence (1: one pass, no scratch memory): as many as make one wave of
// blocks at one an SM, each of at least 128 tokens, and no more than keep the scratch memory under 1 GiB.
extern "C" int plm_decay_chunk_plan(int n_seqs, int H, int N, int P, int max_new, int n_tokens, int* out) {
    out[0] = max_new > 0 ? (max_new + C - 1) / C * C : C;
    out[1] = 1;
    if (n_seqs <= 0 || H <= 0 || N <= 0 || P <= 0) return PLM_ERR_SHAPE;
    if (max_new < 4 * C) return PLM_OK;
    long busy = n_tokens > 0 ? ((long)n_tokens + max_new - 1) / max_new : n_seqs;     // sequences' worth of work
    if (busy > n_seqs) busy = n_seqs;
    if (busy < 1) busy = 1;
    const long blocks = busy * H * ((P + PT - 1) / PT);
    long segs = (long)PLM_SM_COUNT / blocks;
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
// powers [H][65] fp32; state [slots][>= H * N * P] fp32; y [T, H * P] fp32; seg_state for max_segs > 1.  rotate: q and k are
// rotated (half pairs a head, cos and sin [positions][half] fp32, positions tok_pos [T]; half 0: not) and k times k_scale.
extern "C" int plm_decay_chunk_scan(const void* q, const void* k, const void* v, long ldq, long ldk, long ldv, const float* powers,
                                    float* state, long state_stride, float* y, long ldy, const int* seq_start,
                                    const int* seq_slot, int n_seqs, int H, int N, int P, int seg_len, int max_segs,
                                    float* seg_state, int silu, int rotate, const float* cos_t, const float* sin_t,
                                    const int* tok_pos, int half, float k_scale, cudaStream_t stream) {
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
    a.cos_t = cos_t, a.sin_t = sin_t, a.tok_pos = tok_pos, a.half = half, a.k_scale = k_scale;
    if (rotate) {
        if (silu || half < 0 || 2 * half > N || (half > 0 && (!cos_t || !sin_t || !tok_pos))) return PLM_ERR_SHAPE;
        if (((uintptr_t)cos_t | (uintptr_t)sin_t) & 15) return PLM_ERR_ALIGN;
        return N <= 64 ? launch<64, true>(a, stream) : launch<128, true>(a, stream);
    }
    return N <= 64 ? launch<64, false>(a, stream) : launch<128, false>(a, stream);
}

// One token for each of n_seqs sequences (token b of q, k, v is sequence b's): `decay` [H] fp32, the rest as above; any
// element type, N and P (a multiple of 4; state rows and heads on 16-byte boundaries).
extern "C" int plm_decay_step(const void* q, const void* k, const void* v, int dtype, long ldq, long ldk, long ldv,
                              const float* decay, float* state, long state_stride, float* y, long ldy, const int* seq_slot,
                              int n_seqs, int H, int N, int P, int silu, const float* cos_t, const float* sin_t,
                              const int* tok_pos, int half, float k_scale, cudaStream_t stream) {
    if (half < 0 || 2 * half > N || (half > 0 && (silu || !cos_t || !sin_t || !tok_pos))) return PLM_ERR_SHAPE;
    if (n_seqs <= 0 || H <= 0 || N <= 0 || N > 4096 || P <= 0 || P % 4 || n_seqs > 65535 || H > 65535) return PLM_ERR_SHAPE;
    if (((uintptr_t)state & 15) || state_stride % 4) return PLM_ERR_ALIGN;
    const dim3 grid((P + STEP_COLS - 1) / STEP_COLS, H, n_seqs);
    const size_t smem = ((size_t)(2 * N + 3) / 4 * 4 + 16 * STEP_COLS) * sizeof(float);
    if (dtype == PLM_F32)
        return plm_status_of(launch_pdl(decay_step_kernel<float>, grid, dim3(STEP_NT), smem, stream, (const float*)q, (const float*)k,
                                        (const float*)v, ldq, ldk, ldv, decay, state, state_stride, y, ldy, seq_slot, N, P, silu, cos_t, sin_t, tok_pos, half, k_scale));
    if (dtype == PLM_BF16)
        return plm_status_of(launch_pdl(decay_step_kernel<bf16>, grid, dim3(STEP_NT), smem, stream, (const bf16*)q, (const bf16*)k,
                                        (const bf16*)v, ldq, ldk, ldv, decay, state, state_stride, y, ldy, seq_slot, N, P, silu, cos_t, sin_t, tok_pos, half, k_scale));
    return PLM_ERR_DTYPE;
}

// q, k (and with vo, v) [T, H * N] ([T, H * P]) of `dtype` with row strides -> qk [T, 2 H N] and vo [T, H P], fp32: rotated and
// scaled as above.
extern "C" int plm_rotate_rows(const void* q, const void* k, const void* v, int dtype, long ldq, long ldk, long ldv,
                               const float* cos_t, const float* sin_t, const int* tok_pos, int half, float k_scale, float* qk,
                               float* vo, int n_tokens, int H, int N, int P, cudaStream_t stream) {
    if (n_tokens <= 0) return PLM_OK;
    if (H <= 0 || N <= 0 || P <= 0 || half < 0 || 2 * half > N || (half > 0 && (!cos_t || !sin_t || !tok_pos))) return PLM_ERR_SHAPE;
    if (dtype == PLM_F32)
        return plm_status_of(launch_pdl(rotate_rows_kernel<float>, dim3(n_tokens), dim3(256), 0, stream, (const float*)q, (const float*)k,
                                        (const float*)v, ldq, ldk, ldv, cos_t, sin_t, tok_pos, half, k_scale, qk, vo, H, N, P));
    if (dtype == PLM_BF16)
        return plm_status_of(launch_pdl(rotate_rows_kernel<bf16>, dim3(n_tokens), dim3(256), 0, stream, (const bf16*)q, (const bf16*)k,
                                        (const bf16*)v, ldq, ldk, ldv, cos_t, sin_t, tok_pos, half, k_scale, qk, vo, H, N, P));
    return PLM_ERR_DTYPE;
}
