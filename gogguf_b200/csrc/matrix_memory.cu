// A matrix memory per head with exponential gates and a running maximum:
//
//     i = cap tanh(z_i / cap),   f = log sigmoid(cap tanh(z_f / cap))              z: projections with a bias, float32
//     m' = max(f + m, i),   S <- e^(f + m - m') S + e^(i - m') k v^T,   n <- e^(f + m - m') n + e^(i - m') k
//     o = S^T (s q) / (max(|n . (s q)|, e^(-m')) + DEN_EPS),   out = o / sqrt(mean(o^2) + eps) * w * sigmoid(x_g)
//
// S [H][d][dv], n [H][d] and m [H] (float32, all zero at a sequence's start) live in the cache's per-slot states.
// q, k, v and the gate's logits x_g are columns of the projection's row.  Everything between the projections' outputs
// and the stored row is float32.
//
// Two forms.  Token by token: a CTA per (sequence, head) holds the head whole, so the memory's update, the norm over
// the head and the output gate are one kernel (decode steps, short stretches, the 32-bit path).  In chunks (prompts in
// the 16-bit path): see below.
#include "common.cuh"

#define MM_DEN_EPS 1e-6f

__device__ __forceinline__ float mm_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float mm_in_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mm_log_forget(float z, float cap) {        // log sigmoid(u) = min(u, 0) - log(1 + e^-|u|)
    const float u = cap * tanhf(z / cap);
    return fminf(u, 0.f) - log1pf(expf(-fabsf(u)));
}

template <typename T, int V> __device__ __forceinline__ void mm_load(const float* p, float* v) {
    if (V == 4) { const float4 a = *reinterpret_cast<const float4*>(p); v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; }
    else v[0] = p[0];
}
template <int V> __device__ __forceinline__ void mm_store(float* p, const float* v) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
}

#define MM_NT 512

// Thread (part, column group): rows part, part + parts, ... of V neighbouring columns.  RPT > 0: at most RPT rows a
// thread, kept in registers while the sequence's tokens go by (asked for all at once); RPT == 0: heads beyond the
// registers, the state is read and written per token.
template <typename TX, typename T, int V, int RPT>
__global__ void __launch_bounds__(MM_NT) memory_scan_kernel(
    const TX* x, long long ld, int q_off, int k_off, int v_off, int g_off, const float* zi, const float* zf, long long ldz,
    T* out, float* S_state, float* n_state, float* m_state, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
    const int* __restrict__ seq_of_token, const float* __restrict__ w, int H, int d, int dv, int groups, int parts, float q_scale,
    float cap, float eps) {
    pdl_launch();
    pdl_wait();
    extern __shared__ float sm[];
    const int b = blockIdx.x, h = blockIdx.y;
    const int start = cu_seqlens[b], end = cu_seqlens[b + 1];
    if (end <= start) return;
    const size_t HV = (size_t)H * dv;
    if (seq_of_token[start] < 0) {
        for (int t = start; t < end; ++t)
            for (int j = threadIdx.x; j < dv; j += MM_NT) out[(size_t)t * HV + (size_t)h * dv + j] = from_f<T>(0.f);
        return;
    }
    float* red = sm;                          // [40]
    float* qs = red + 40;                     // [d]
    float* ks = qs + d;                       // [d]
    float* ns = ks + d;                       // [d]
    float* vs = ns + d + ((4 - (3 * d) % 4) % 4);      // [dv], on a 16-byte boundary
    float* os = vs + dv + ((4 - dv % 4) % 4);          // [parts][dv]
    const int slot = slots[b];
    float* Sp = S_state + ((size_t)slot * H + h) * d * dv;
    float* np = n_state + ((size_t)slot * H + h) * d;
    const int part = threadIdx.x / groups, col = (threadIdx.x - part * groups) * V;
    const bool live = part < parts;
    float R[RPT > 0 ? RPT * V : 1];
    if (RPT > 0 && live) {
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int r = part + i * parts;
            if (r < d) mm_load<T, V>(Sp + (size_t)r * dv + col, R + i * V);
        }
    }
    for (int r = threadIdx.x; r < d; r += MM_NT) ns[r] = np[r];
    float m = m_state[(size_t)slot * H + h];
    for (int t = start; t < end; ++t) {
        const TX* row = x + (size_t)t * ld;
        float den = 0.f;
        const float li = mm_in_gate(zi[(size_t)t * ldz + h], cap), lf = mm_log_forget(zf[(size_t)t * ldz + h], cap);
        const float mn = fmaxf(lf + m, li), keep = expf(lf + m - mn), add = expf(li - mn);
        m = mn;
        __syncthreads();                       // the token before is done with q, k, v and the partial sums
        for (int r = threadIdx.x; r < d; r += MM_NT) {
            const float q = to_f<TX>(row[q_off + h * d + r]) * q_scale, k = to_f<TX>(row[k_off + h * d + r]);
            qs[r] = q;
            ks[r] = add * k;
            const float n = fmaf(keep, ns[r], add * k);
            ns[r] = n;
            den = fmaf(n, q, den);
        }
        for (int j = threadIdx.x; j < dv; j += MM_NT) vs[j] = to_f<TX>(row[v_off + h * dv + j]);
        den = block_sum(den, red);             // (its barriers also order q, k and v before their use)
        if (live) {
            float acc[V], vv[V];
#pragma unroll
            for (int e = 0; e < V; ++e) { acc[e] = 0.f; vv[e] = vs[col + e]; }
            if (RPT > 0) {
#pragma unroll
                for (int i = 0; i < RPT; ++i) {
                    const int r = part + i * parts;
                    if (r < d) {
                        const float kk = ks[r], qq = qs[r];
#pragma unroll
                        for (int e = 0; e < V; ++e) {
                            R[i * V + e] = fmaf(keep, R[i * V + e], kk * vv[e]);
                            acc[e] = fmaf(R[i * V + e], qq, acc[e]);
                        }
                    }
                }
            } else {
#pragma unroll 8
                for (int r = part; r < d; r += parts) {
                    float s[V];
                    mm_load<T, V>(Sp + (size_t)r * dv + col, s);
                    const float kk = ks[r], qq = qs[r];
#pragma unroll
                    for (int e = 0; e < V; ++e) { s[e] = fmaf(keep, s[e], kk * vv[e]); acc[e] = fmaf(s[e], qq, acc[e]); }
                    mm_store<V>(Sp + (size_t)r * dv + col, s);
                }
            }
            mm_store<V>(os + (size_t)part * dv + col, acc);
        }
        __syncthreads();
        const float inv = 1.0f / (fmaxf(fabsf(den), expf(-mn)) + MM_DEN_EPS);
        float ss = 0.f;
        for (int j = threadIdx.x; j < dv; j += MM_NT) {
            float o = 0.f;
            for (int p = 0; p < parts; ++p) o += os[(size_t)p * dv + j];
            o *= inv;
            vs[j] = o;                         // (nobody reads v any more: the barrier above)
            ss = fmaf(o, o, ss);
        }
        ss = block_sum(ss, red);
        const float f = 1.0f / sqrtf(ss / (float)dv + eps);
        for (int j = threadIdx.x; j < dv; j += MM_NT)      // the thread that wrote vs[j] reads it
            out[(size_t)t * HV + (size_t)h * dv + j] =
                from_f<T>(vs[j] * f * w[h * dv + j] * mm_sigmoid(to_f<TX>(row[g_off + h * dv + j])));
    }
    if (RPT > 0 && live) {
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int r = part + i * parts;
            if (r < d) mm_store<V>(Sp + (size_t)r * dv + col, R + i * V);
        }
    }
    for (int r = threadIdx.x; r < d; r += MM_NT) np[r] = ns[r];          // (a thread's own rows throughout)
    if (threadIdx.x == 0) m_state[(size_t)slot * H + h] = m;
}

// x [T, ld] in `x_dtype`: q and k heads (H d columns each) at q_off and k_off, v heads and the output gate's logits (H dv
// each) at v_off and g_off; zi, zf float32, rows ldz apart (H columns each); out [T, H dv] in `dtype`; w [H dv].
GG_API gg_memory_scan(const void* x, int x_dtype, long long ld, int q_off, int k_off, int v_off, int g_off, const float* zi,
                      const float* zf, long long ldz, void* out, int dtype, float* S_state, float* n_state, float* m_state,
                      const int* cu_seqlens, const int* slots, const int* seq_of_token, const float* w, int ntok, int n_seqs, int H,
                      int d, int dv, float q_scale, float cap, float eps, cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0) return 0;
    if (H <= 0 || H > 65535 || d <= 0 || dv <= 0 || !(cap > 0.f) || S_state == nullptr || n_state == nullptr || m_state == nullptr ||
        w == nullptr || zi == nullptr || zf == nullptr)
        return GG_ERR_ARG;
    const bool vec = dv % 4 == 0 && (((uintptr_t)S_state) & 15) == 0;
    const int groups = vec ? dv / 4 : dv;
    if (groups > MM_NT) return GG_ERR_ARG;
    int parts = MM_NT / groups;
    if (parts > d) parts = d;
    const int rows = (d + parts - 1) / parts;
    const size_t smem = ((size_t)40 + 3 * d + 4 + dv + 4 + (size_t)parts * dv) * sizeof(float);
    if (smem > 200 * 1024) return GG_ERR_ARG;
#define GG_MM(TX_, T_, V_, R_)                                                                                           \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            cudaFuncSetAttribute(memory_scan_kernel<TX_, T_, V_, R_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        gg_launch(memory_scan_kernel<TX_, T_, V_, R_>, dim3(n_seqs, H), dim3(MM_NT), smem, stream, 1, (const TX_*)x, ld, q_off,  \
                  k_off, v_off, g_off, zi, zf, ldz, (T_*)out, S_state, n_state, m_state, cu_seqlens, slots, seq_of_token, w, H, d, \
                  dv, groups, parts, q_scale, cap, eps);                                                                 \
    } while (0)
    GG_DISPATCH_DTYPE(dtype, T,
        GG_DISPATCH_DTYPE(x_dtype, TX,
            if (vec) {
                if (rows > 16) GG_MM(TX, T, 4, 0);
                else if (rows <= 4) GG_MM(TX, T, 4, 4);
                else if (rows <= 8) GG_MM(TX, T, 4, 8);
                else GG_MM(TX, T, 4, 16);
            } else {
                if (rows > 64) GG_MM(TX, T, 1, 0);
                else if (rows <= 16) GG_MM(TX, T, 1, 16);
                else GG_MM(TX, T, 1, 64);
            }));
#undef GG_MM
    return gg_last_error();
}
