// Attention with mixed heads (see mixed_head_attention.cu) of prompts on the 5th-generation tensor cores.
//
// One CTA per (128 query rows of one sequence, query head, NV kv heads' values).  Per 64-key page S = Q K^T
// (tcgen05.mma 128 x 64 x 16, Q and K as K-major tiles staged by TMA) lands in tensor memory; four softmax warps
// read it, one query row per thread, apply the query's temperature, the bound and the mask, and write P as bfloat16
// back over the first half of the score buffer; U_n += P V_n (P as the A operand straight from tensor memory, V_n as the
// MN-major B operand) accumulates in tensor memory for each of the CTA's kv heads n.  The results leave unnormalised,
// u [row of the step][head][kv head][dv] with each row's reference (log2 units) and sum, ml [row][head][2]; the combining
// kernel of mixed_head_attention.cu divides, mixes and gates.
//
// The reference that P and the row sum are taken against need not be a maximum (the result is exact whatever it is, as
// long as nothing overflows).  Scores bounded by c lie in [-c, c], so a modest bound needs none: zero serves.  Otherwise
// a page is computed against the reference of the pages before it, and only when its sum says that a score lies more than
// 2^64 above it (or the row has none yet) does the warp find the page's maximum, rescale U where it has grown by more
// than 2^8, and compute the page again.
//
// The bound is c tanh(x), x = s / c.  Where a page's |x| stay below one in all of a warp's rows (the usual case) tanh is
// x p(x^2) with p of degree six, a Chebyshev fit of tanh(sqrt t) / sqrt t on [0, 1] (absolute error below 1.5e-7), two
// numbers per instruction on the multiply-add pipe; otherwise one exponential and one division per score.
#include "tma_util.cuh"

#define MHP_PAGE 64
#define MHP_MODEST 57.0f          // a bound (log2 units) below this keeps the sum of 64 weights below 2^64
#define MHP_LOG2E 1.4426950408889634f

namespace {

__device__ __forceinline__ float mhp_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void mhp_store8(float* dst, const uint32_t* r) {
    asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(dst), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]),
                 "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]) : "memory");
}
typedef unsigned long long f2;
__device__ __forceinline__ f2 pk2(float lo, float hi) {
    f2 v;
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
    return v;
}
__device__ __forceinline__ void un2(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
    f2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
    f2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f2 add2(f2 a, f2 b) {
    f2 d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint32_t mhp_bf2(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

template <int D, int DV, int NV>
struct PromptSizes {
    static constexpr int QBOX = 128 * 64 * 2, KBOX = 64 * 64 * 2;          // bytes of a 64-column box of Q, of K or V
    static constexpr int QH = D / 64, VH = DV / 64;
    static constexpr int Q_BYTES = QH * QBOX, K_STAGE = QH * KBOX, V_HEAD = VH * KBOX, V_STAGE = NV * V_HEAD;
    static constexpr int SMEM = Q_BYTES + 2 * K_STAGE + 2 * V_STAGE + 256;
    static constexpr int COLS = 128 + NV * DV;                              // two score buffers, then the accumulators
    static constexpr int TMEM = COLS <= 256 ? 256 : 512;
};

// GROUPS softmax warpgroups.  One: any scores.  Two (scores that need no running reference): both take every page, 32 of
// its 64 keys each.  Four: two such pairs take turns, the even pages and the odd ones, each with a score buffer of its own.
template <int D, int DV, int NV, int GROUPS>
__global__ void __launch_bounds__(GROUPS * 128 + 64, PromptSizes<D, DV, NV>::TMEM == 256 ? 2 : 1) mixed_head_prompt_kernel(
    const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
    float* __restrict__ u, float* __restrict__ ml, const int* __restrict__ cu_seqlens, const int* __restrict__ ctx_lens,
    const int* __restrict__ seq_of_token, const int* __restrict__ page_table, int max_pages, int n_seqs, int H, int G, int d,
    int dv, float scale, float cap, float coef, float every, int window, int n_pages, int* __restrict__ status) {
    typedef PromptSizes<D, DV, NV> Z;
    constexpr int SW = GROUPS * 4;                  // softmax warps; then the TMA warp and the MMA warp
    constexpr bool PAIR = GROUPS > 1;               // no reference is kept
    constexpr int STEP = GROUPS == 4 ? 2 : 1, NK = PAIR ? 32 : 64;      // pages from one of a thread's to its next, keys of it
    extern __shared__ __align__(1024) uint8_t smem[];
    uint8_t* Qs = smem;
    uint8_t* Ks = Qs + Z::Q_BYTES;                  // two stages
    uint8_t* Vs = Ks + 2 * Z::K_STAGE;              // two stages of NV heads
    uint64_t* bars = (uint64_t*)(Vs + 2 * Z::V_STAGE);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;                    // [2]
    uint64_t* k_empty = bars + 3;                   // [2]
    uint64_t* v_full = bars + 5;                    // [2]
    uint64_t* v_empty = bars + 7;                   // [2]
    uint64_t* s_full = bars + 9;                    // [2]
    uint64_t* p_ready = bars + 11;                  // [2]: a softmax warp may be a page ahead of another
    uint64_t* pv_done = bars + 13;
    uint64_t* u_done = bars + 14;                   // every P V is complete
    uint32_t* tmem_slot = (uint32_t*)(bars + 15);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

    // no early release of the next kernel: see the note on dependent launches in common.cuh
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        tma::mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) {
            tma::mbar_init(&k_full[i], 1); tma::mbar_init(&k_empty[i], 1);
            tma::mbar_init(&v_full[i], 1); tma::mbar_init(&v_empty[i], 1);
            tma::mbar_init(&s_full[i], 1);
            tma::mbar_init(&p_ready[i], PAIR ? 8 : 4);       // one arrival per softmax warp of the page
        }
        tma::mbar_init(pv_done, 1);
        tma::mbar_init(u_done, 1);
        *abort_flag = 0;
        tma::mbar_fence_init();
        tma::prefetch_map(&tmQ); tma::prefetch_map(&tmK); tma::prefetch_map(&tmV);
    }
    if (warp == SW + 1) tc5::alloc(tmem_slot, Z::TMEM);
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_wait();

    // which (sequence, 128-row query tile)?  heavy tiles (late rows) first
    int b = -1, tile = (int)gridDim.y - 1 - (int)blockIdx.y, n_new = 0, tok0 = 0;
    for (int i = 0; i < n_seqs; ++i) {
        const int a = cu_seqlens[i], e = cu_seqlens[i + 1];
        if (e <= a || seq_of_token[a] < 0) continue;
        const int nt = (e - a + 127) >> 7;
        if (tile < nt) { b = i; n_new = e - a; tok0 = a; break; }
        tile -= nt;
    }
    const bool aligned = (tma::smem_u32(smem) & 1023u) == 0;     // (the swizzled tiles need it)
    if (!aligned && threadIdx.x == 0) atomicCAS(status, 0, 69);
    const bool active = b >= 0 && aligned;
    const int h = blockIdx.x % H, v0 = (blockIdx.x / H) * NV;
    const int nv = min(NV, G - v0);
    const int kvh = h / (H / G);
    const int row0 = tile * 128;
    const int rows = active ? min(128, n_new - row0) : 0;
    const int pos0 = active ? ctx_lens[b] - n_new + row0 : 0;
    const int lo = (window > 0 && pos0 - window + 1 > 0) ? pos0 - window + 1 : 0;
    const int kt_first = lo / MHP_PAGE, kt_last = active ? (pos0 + rows - 1) / MHP_PAGE : -1;
    const int ntiles = active ? kt_last - kt_first + 1 : 0;
    const uint32_t S_t = tmem_base, U_t = tmem_base + 128;

    if (warp == SW) {
        if (lane == 0 && active) {
            const int* pt = page_table + (size_t)b * max_pages;
            tma::mbar_expect_tx(q_full, Z::Q_BYTES);
#pragma unroll
            for (int hf = 0; hf < Z::QH; ++hf) tma::load_2d(Qs + hf * Z::QBOX, &tmQ, q_full, h * d + hf * 64, tok0 + row0);
            auto page_of = [&](int j) { return gg_page(pt, kt_first + j, max_pages, PageBounds{n_pages, status}, 53); };
            int next = ntiles > 0 ? page_of(0) : 0;
            for (int j = 0; j < ntiles; ++j) {
                const int s = j & 1;
                const uint32_t ph = (uint32_t)((j >> 1) & 1) ^ 1u;
                const int page = next;
                if (j + 1 < ntiles) next = page_of(j + 1);     // (on its way while this page's places come free)
                if (!tma::mbar_wait(&k_empty[s], ph, abort_flag, status, 61)) break;
                tma::mbar_expect_tx(&k_full[s], Z::K_STAGE);
#pragma unroll
                for (int hf = 0; hf < Z::QH; ++hf)
                    tma::load_2d(Ks + s * Z::K_STAGE + hf * Z::KBOX, &tmK, &k_full[s], hf * 64, (page * G + kvh) * MHP_PAGE);
                if (!tma::mbar_wait(&v_empty[s], ph, abort_flag, status, 62)) break;
                tma::mbar_expect_tx(&v_full[s], nv * Z::V_HEAD);
#pragma unroll
                for (int n = 0; n < NV; ++n) {
                    if (n >= nv) break;
#pragma unroll
                    for (int hf = 0; hf < Z::VH; ++hf)
                        tma::load_2d(Vs + s * Z::V_STAGE + n * Z::V_HEAD + hf * Z::KBOX, &tmV, &v_full[s], hf * 64,
                                     (page * G + v0 + n) * MHP_PAGE);
                }
            }
        }
    } else if (warp == SW + 1) {
        // All lanes walk the loop together, so that addresses and descriptors stay uniform; one elected lane issues.
        if (active) {
            const uint32_t idesc_qk = tc5::idesc_bf16(128, 64, 0), idesc_pv = tc5::idesc_bf16(128, DV, 1);
            const uint64_t q_d = tc5::smem_desc(tma::smem_u32(Qs), 16, 1024), k_d = tc5::smem_desc(tma::smem_u32(Ks), 16, 1024);
            const uint64_t v_d = tc5::smem_desc(tma::smem_u32(Vs), Z::KBOX, 1024);
            auto await = [&](uint64_t* bar, int j, int code) -> bool {      // (a lane that gives up takes the others with it)
                return __all_sync(0xffffffffu, tma::mbar_wait(bar, (uint32_t)((j >> 1) & 1), abort_flag, status, code));
            };
            auto issue_scores = [&](int j) -> bool {            // scores of page j into buffer j & 1
                const int s = j & 1;
                if (!await(&k_full[s], j, 64)) return false;
                tc5::fence_after();
                const uint64_t kd = k_d + (uint64_t)(s * (Z::K_STAGE >> 4));
                if (tc5::elect_one()) {
#pragma unroll
                    for (int ks = 0; ks < D / 16; ++ks) {
                        const uint64_t qo = (uint64_t)(((ks >> 2) * Z::QBOX + (ks & 3) * 32) >> 4);
                        const uint64_t ko = (uint64_t)(((ks >> 2) * Z::KBOX + (ks & 3) * 32) >> 4);
                        tc5::mma(S_t + (uint32_t)(s * 64), q_d + qo, kd + ko, idesc_qk, ks > 0 ? 1u : 0u);
                    }
                    tc5::commit(&s_full[s]);
                    tc5::commit(&k_empty[s]);
                }
                __syncwarp();
                return true;
            };
            bool ok = await(q_full, 0, 63);
            if (ok && ntiles > 0) ok = issue_scores(0);
            for (int j = 0; j < ntiles && ok; ++j) {
                // the next page's scores: their buffer was last read by the softmax of page j - 1, whose p_ready this
                // warp has seen, and by the P V of page j - 1, which was issued before them
                if (j + 1 < ntiles && !(ok = issue_scores(j + 1))) break;
                const int s = j & 1;
                if (!(ok = await(&v_full[s], j, 66))) break;
                if (!(ok = await(&p_ready[s], j, 65))) break;
                tc5::fence_after();
                const uint64_t vd = v_d + (uint64_t)(s * (Z::V_STAGE >> 4));
                const uint32_t pa = S_t + (uint32_t)(s * 64), first = j > 0 ? 1u : 0u;
                if (tc5::elect_one()) {
#pragma unroll
                    for (int n = 0; n < NV; ++n) {
                        if (n >= nv) break;
#pragma unroll
                        for (int kk = 0; kk < 4; ++kk)
                            // (16 keys of P are 8 columns; each group's lie over the scores it alone has read)
                            tc5::mma_a_tmem(U_t + (uint32_t)(n * DV), pa + (uint32_t)(PAIR ? (kk >> 1) * 32 + (kk & 1) * 8 : kk * 8),
                                            vd + (uint64_t)((n * Z::V_HEAD + kk * 2048) >> 4), idesc_pv, kk > 0 ? 1u : first);
                    }
                    tc5::commit(pv_done);
                    tc5::commit(&v_empty[s]);
                }
                __syncwarp();
            }
            if (ok && tc5::elect_one()) tc5::commit(u_done);
            __syncwarp();
        }
    } else if (active) {
        const int row = threadIdx.x & 127;                 // query row of the tile = tensor-memory lane
        const int wg = warp >> 2, half = PAIR ? wg & 1 : 0;      // (of a page's keys)
        const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
        const int p = pos0 + row;
        const float tau = coef == 0.f ? 1.0f : 1.0f + coef * logf(floorf((float)(p + 1) / every) + 1.0f);
        const float fac = scale * tau * (cap > 0.f ? 1.0f / cap : MHP_LOG2E);
        const float cap_log2 = cap * MHP_LOG2E;
        const f2 fac2 = pk2(fac, fac);
        // the reference in use (log2 units); a bound that keeps 64 weights below 2^64 needs none
        float ref = (cap > 0.f && cap_log2 < MHP_MODEST) ? 0.f : -INFINITY;
        float l = 0.f;
        bool ok = true;
        for (int j = GROUPS == 4 ? wg >> 1 : 0; j < ntiles; j += STEP) {
            if (!tma::mbar_wait(&s_full[j & 1], (uint32_t)((j >> 1) & 1), abort_flag, status, 67)) { ok = false; break; }
            tc5::fence_after();
            uint32_t sr[NK];
            tc5::ld32(S_t + lane_off + (uint32_t)((j & 1) * 64 + half * 32), sr);
            if (!PAIR) tc5::ld32(S_t + lane_off + (uint32_t)((j & 1) * 64) + 32, sr + (NK - 32));
            tc5::wait_ld();
            auto pair = [&](int e) { return pk2(__uint_as_float(sr[2 * e]), __uint_as_float(sr[2 * e + 1])); };
            auto put = [&](int e, f2 v) {
                float a, c;
                un2(v, a, c);
                sr[2 * e] = __float_as_uint(a);
                sr[2 * e + 1] = __float_as_uint(c);
            };
#pragma unroll
            for (int e = 0; e < NK / 2; ++e) put(e, mul2(pair(e), fac2));
            if (cap > 0.f) {
                float mx4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int c = 0; c < NK; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], fabsf(__uint_as_float(sr[c])));
                const bool wide = !(fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) <= 1.0f);
                if (!__any_sync(0xffffffffu, wide)) {
                    const float cf[7] = {0.9999999403953552f, -0.33332857489585876f, 0.13325397670269012f, -0.05346517637372017f,
                                         0.020305519923567772f, -0.006217069923877716f, 0.0010455535957589746f};
                    constexpr int RUN = 8;                 // pairs side by side: the chains of multiply-adds overlap
#pragma unroll
                    for (int e0 = 0; e0 < NK / 2; e0 += RUN) {
                        f2 t[RUN], q[RUN];
#pragma unroll
                        for (int e = 0; e < RUN; ++e) { t[e] = mul2(pair(e0 + e), pair(e0 + e)); q[e] = pk2(cf[6] * cap_log2, cf[6] * cap_log2); }
#pragma unroll
                        for (int k = 5; k >= 0; --k) {
                            const f2 ck = pk2(cf[k] * cap_log2, cf[k] * cap_log2);
#pragma unroll
                            for (int e = 0; e < RUN; ++e) q[e] = fma2(t[e], q[e], ck);
                        }
#pragma unroll
                        for (int e = 0; e < RUN; ++e) put(e0 + e, mul2(pair(e0 + e), q[e]));
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < NK; ++c) {
                        const float t = mhp_ex2(__uint_as_float(sr[c]) * (2.0f * MHP_LOG2E));
                        sr[c] = __float_as_uint(cap_log2 - __fdividef(2.0f * cap_log2, t + 1.0f));
                    }
                }
            }
            const int key0 = (kt_first + j) * MHP_PAGE;
            if ((key0 + MHP_PAGE - 1 > pos0) || (window > 0 && key0 < pos0 + 127 - window + 1)) {
#pragma unroll
                for (int c = 0; c < NK; ++c) {
                    const int kidx = key0 + half * 32 + c;
                    if (!(kidx <= p && (window <= 0 || kidx > p - window))) sr[c] = 0xff800000u;
                }
            }
            uint32_t pb[NK / 2];
            auto exponentials = [&]() -> float {           // P against the reference in use; returns the page's sum
                const float mu = ref == -INFINITY ? 0.f : ref;
                const f2 nmu = pk2(-mu, -mu);
                f2 l4[4] = {pk2(0.f, 0.f), pk2(0.f, 0.f), pk2(0.f, 0.f), pk2(0.f, 0.f)};
#pragma unroll
                for (int e = 0; e < NK / 2; ++e) {
                    float x0, x1;
                    un2(PAIR ? pair(e) : add2(pair(e), nmu), x0, x1);
                    const float p0 = mhp_ex2(x0), p1 = mhp_ex2(x1);
                    l4[e & 3] = add2(l4[e & 3], pk2(p0, p1));
                    pb[e] = mhp_bf2(p0, p1);
                }
                float la, lb;
                un2(add2(add2(l4[0], l4[1]), add2(l4[2], l4[3])), la, lb);
                return la + lb;
            };
            float lpage = 0.f;
            if (PAIR) {
                lpage = exponentials();
            } else {
                bool again = ref == -INFINITY;
                if (!__any_sync(0xffffffffu, again)) {
                    lpage = exponentials();
                    again = !(lpage < 1.8446744e19f);
                }
                if (__any_sync(0xffffffffu, again)) {
                    float m8[8];
#pragma unroll
                    for (int k = 0; k < 8; ++k) m8[k] = __uint_as_float(sr[k]);
#pragma unroll
                    for (int c = 8; c < NK; ++c) m8[c & 7] = fmaxf(m8[c & 7], __uint_as_float(sr[c]));
                    const float mx = fmaxf(fmaxf(fmaxf(m8[0], m8[1]), fmaxf(m8[2], m8[3])), fmaxf(fmaxf(m8[4], m8[5]), fmaxf(m8[6], m8[7])));
                    const bool grow = mx > ref + 8.0f || (ref == -INFINITY && mx != -INFINITY);
                    if (__any_sync(0xffffffffu, grow)) {
                        float corr = 1.0f;
                        if (grow) {
                            corr = ref == -INFINITY ? 0.f : mhp_ex2(ref - mx);
                            ref = mx;
                            l *= corr;
                        }
                        if (j > 0) {                           // P V of the page before must be complete before U is rescaled
                            if (!tma::mbar_wait(pv_done, (uint32_t)((j - 1) & 1), abort_flag, status, 68)) { ok = false; break; }
                            tc5::fence_after();
#pragma unroll 1
                            for (int c0 = 0; c0 < nv * DV; c0 += 32) {
                                uint32_t orow[32];
                                tc5::ld32(U_t + lane_off + c0, orow);
                                tc5::wait_ld();
#pragma unroll
                                for (int c = 0; c < 32; ++c) orow[c] = __float_as_uint(__uint_as_float(orow[c]) * corr);
                                tc5::st32(U_t + lane_off + c0, orow);
                            }
                            tc5::wait_st();
                        }
                    }
                    lpage = exponentials();
                }
            }
            l += lpage;
            // P over this thread's own row of the scores it has read: the P V that read the P of two pages ago from this
            // buffer was issued before these scores, and the tensor core works in order
            if constexpr (PAIR) tc5::st16(S_t + lane_off + (uint32_t)((j & 1) * 64 + half * 32), pb);
            else tc5::st32(S_t + lane_off + (uint32_t)((j & 1) * 64), pb);
            tc5::wait_st();
            tc5::fence_before();
            __syncwarp();
            if (lane == 0) tma::mbar_arrive(&p_ready[j & 1]);
        }
        ok = ok && tma::mbar_wait(u_done, 0, abort_flag, status, 68);
        const size_t at = (size_t)(tok0 + row0 + row) * H + h;
        if (PAIR) {
            // the groups' sums of a row come together (all of them come here, whatever happened to their waits)
            float* sums = reinterpret_cast<float*>(smem);   // (Q is not read any more: its last reader is complete, or nothing is)
            if (wg > 0) sums[(wg - 1) * 128 + row] = l;
            asm volatile("bar.sync 1, %0;" :: "n"(GROUPS * 128) : "memory");
            if (wg == 0)
                for (int k = 0; k < GROUPS - 1; ++k) l += sums[k * 128 + row];
        }
        if (ok) {
            tc5::fence_after();
            if (row < rows && v0 == 0 && wg == 0) { ml[at * 2] = ref; ml[at * 2 + 1] = l; }
            // (the warpgroups share the runs of 32 columns out)
#pragma unroll 1
            for (int c0 = 32 * wg; c0 < nv * DV; c0 += 32 * GROUPS) {
                const int n = c0 / DV, e0 = c0 % DV;
                float* dst = u + (at * G + v0 + n) * dv + e0;
                uint32_t orow[32];
                tc5::ld32(U_t + lane_off + (uint32_t)c0, orow);
                tc5::wait_ld();
                if (row < rows) {
#pragma unroll
                    for (int c = 0; c < 32; c += 8)            // (dv is a multiple of 8: whole sectors of 32 bytes)
                        if (e0 + c < dv) mhp_store8(dst + c, orow + c);
                }
            }
        }
    }
    tc5::fence_before();
    __syncthreads();
    if (*abort_flag) {                                     // let what is in flight land before the memory goes back
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) { }
        __syncthreads();
    }
    if (warp == SW + 1) {
        tc5::fence_after();
        tc5::dealloc(tmem_base, Z::TMEM);
    }
}

template <int D, int DV, int NV, int GROUPS>
int launch_prompt_form(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, float* u, float* ml, const int* cu_seqlens,
                  const int* ctx_lens, const int* seq_of_token, const int* page_table, int max_pages, int n_seqs, int max_tiles,
                  int H, int G, int d, int dv, float scale, float cap, float coef, float every, int window, int n_pages,
                  int* status, cudaStream_t stream) {
    auto kern = mixed_head_prompt_kernel<D, DV, NV, GROUPS>;
    constexpr int smem = PromptSizes<D, DV, NV>::SMEM;
    static bool configured = false;                        // per instantiation
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return gg_launch(kern, dim3(H * ((G + NV - 1) / NV), max_tiles), dim3(GROUPS * 128 + 64), smem, stream, 1, tq, tk, tv, u, ml, cu_seqlens,
                     ctx_lens, seq_of_token, page_table, max_pages, n_seqs, H, G, d, dv, scale, cap, coef, every, window, n_pages,
                     status);
}

template <int D, int DV, int NV, typename... Args>
int launch_prompt(bool no_reference, Args... args) {
    // forms that fill tensor memory have the multiprocessor to themselves, the others share it between two CTAs
    if (no_reference) return launch_prompt_form<D, DV, NV, PromptSizes<D, DV, NV>::TMEM == 512 ? 4 : 2>(args...);
    return launch_prompt_form<D, DV, NV, 1>(args...);
}

}  // namespace

// 1 if the kernel takes these sizes.
GG_API gg_mixed_head_prompt_takes(int H, int G, int d, int dv, int page_size) {
    return (d > 0 && d <= 128 && d % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0 && page_size == MHP_PAGE && G > 0 && H % G == 0) ? 1 : 0;
}

// row [ntok, ld] bfloat16 with q [H][d] at column 0; pools k [page][G][64][d], v [..][dv]; u [ntok][H][G][dv] and
// ml [ntok][H][2] float32; max_tiles >= sum over sequences of ceil(new tokens / 128).  cap 0: scores not bounded; coef 0: no
// temperature; window <= 0: none.  value_heads: kv heads' values per CTA (1 or 2; 4 for dv <= 64).  A wait that runs out leaves one of the
// codes 61-68 in the status word.
GG_API gg_mixed_head_prompt(const void* row, long long ld, const void* k_pool, const void* v_pool, float* u, float* ml,
                            const int* cu_seqlens, const int* ctx_lens, const int* seq_of_token, const int* page_table,
                            int max_pages, int page_size, int n_pages, int ntok, int n_seqs, int max_tiles, int H, int G, int d,
                            int dv, float scale, float cap, float coef, float every, int window, int value_heads, int* status,
                            cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0 || max_tiles <= 0) return 0;
    if (!gg_mixed_head_prompt_takes(H, G, d, dv, page_size) || max_tiles > 65535 || n_pages <= 0 || status == nullptr || u == nullptr ||
        ml == nullptr || (ld % 8) || ld < (long long)H * d || cap < 0.f || (coef != 0.f && !(every > 0.f)) ||
        (value_heads != 1 && value_heads != 2 && !(value_heads == 4 && dv <= 64)) ||
        (((uintptr_t)row | (uintptr_t)k_pool | (uintptr_t)v_pool) & 15) || (((uintptr_t)u) & 31))
        return GG_ERR_ARG;
    CUtensorMap tq, tk, tv;
    int rc;
    const unsigned long long rows = (unsigned long long)n_pages * G * MHP_PAGE;
    // (a head narrower than its 64 or 128 columns: the columns of K beyond d are filled with zeros, so that what Q's box
    // holds beyond its head, its neighbour's columns, meets zeros)
    if ((rc = tma::make_map_bf16(&tq, row, (unsigned long long)ntok, H * d, ld, 128)) != 0) return rc;
    if ((rc = tma::make_map_bf16(&tk, k_pool, rows, d, d, MHP_PAGE)) != 0) return rc;
    if ((rc = tma::make_map_bf16(&tv, v_pool, rows, dv, dv, MHP_PAGE)) != 0) return rc;
#define MHP_ARGS cap > 0.f && cap * MHP_LOG2E < MHP_MODEST, tq, tk, tv, u, ml, cu_seqlens, ctx_lens, seq_of_token, page_table, \
        max_pages, n_seqs, max_tiles, H, G, d, dv, scale, cap, coef, every, window, n_pages, status, stream
#define MHP_GO(D_, V_) (value_heads == 2 ? launch_prompt<D_, V_, 2>(MHP_ARGS) : launch_prompt<D_, V_, 1>(MHP_ARGS))
    if (value_heads == 4) return d <= 64 ? launch_prompt<64, 64, 4>(MHP_ARGS) : launch_prompt<128, 64, 4>(MHP_ARGS);
    if (d <= 64) return dv <= 64 ? MHP_GO(64, 64) : MHP_GO(64, 128);
    return dv <= 64 ? MHP_GO(128, 64) : MHP_GO(128, 128);
#undef MHP_ARGS
#undef MHP_GO
}

// 1 if this library was built with checked page tables (the debug build), else 0.
GG_API gg_mixed_head_prompt_checked() { return gg_debug_bounds(); }
