// Between an attention's projections and its paged attention kernel, for attentions whose q, k and v pass a short causal
// convolution over time and whose q and k heads are normed one by one:
//   y[t] = sum_j taps[:, j] * u[t - K + 1 + j]      u: the projected row [q | k | v], channel by channel; before a step's
//                                                   first token of a request come the inputs the request kept (zero for a
//                                                   new request)
//   q, k heads: y / sqrt(mean(y^2) + eps)           without a weight; can be left out
//   q heads:    times 1 + coef * ln((p + 1) / every + 1), the quotient without its remainder, p the position
//   q heads to a buffer of heads padded to D with zeros, k and v heads (padded) into the cache's pages.
// A warp owns one head and walks a run of neighbouring tokens of the packed step with the last K - 1 inputs of its
// channels in registers (K up to 4; longer filters read them again).  A run that would begin among the first K - 1 tokens
// of a segment, but not at its first, leaves those tokens to the run before it: so the kept inputs are read by one warp,
// the one that has the segment's first token, and that warp leaves the segment's last K - 1 inputs in their place.
// The kept inputs of a request: K - 1 rows of [q | k | v] channels, oldest first, float32.
#include "common.cuh"

struct ConvPrepArgs {
    const void* proj; int ld;
    const void* taps; int taps_dtype, K;
    float* kept; long long kept_stride; int kept_off;
    const int* pos; const int* tok_seg; const int* cu_q; const int* seg_slot; const int* block_table; int bt_stride, page_size;
    void* kpool; void* vpool; void* q_out;
    int T, Hq, Hkv, dim, vdim, D, own_kv, write_kv, normed;
    float eps, temp_coef; int temp_every;                  // temp_every 0: no temperature
    int run;
};

template <typename TA, int N>
__device__ __forceinline__ void ld_vec(const TA* p, float (&v)[N]);
template <> __device__ __forceinline__ void ld_vec<float, 1>(const float* p, float (&v)[1]) { v[0] = *p; }
template <> __device__ __forceinline__ void ld_vec<bf16, 1>(const bf16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
template <> __device__ __forceinline__ void ld_vec<bf16, 2>(const bf16* p, float (&v)[2]) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x; v[1] = f.y;
}
template <> __device__ __forceinline__ void ld_vec<bf16, 4>(const bf16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <> __device__ __forceinline__ void ld_vec<bf16, 8>(const bf16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
template <typename TA, int N>
__device__ __forceinline__ void st_vec(TA* p, const float (&v)[N]);
template <> __device__ __forceinline__ void st_vec<float, 1>(float* p, const float (&v)[1]) { *p = v[0]; }
template <> __device__ __forceinline__ void st_vec<bf16, 1>(bf16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
template <> __device__ __forceinline__ void st_vec<bf16, 2>(bf16* p, const float (&v)[2]) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}
template <> __device__ __forceinline__ void st_vec<bf16, 4>(bf16* p, const float (&v)[4]) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
}
template <> __device__ __forceinline__ void st_vec<bf16, 8>(bf16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// KT: filter length held in registers (1 .. 4), or 0 for any length.  A lane holds NI groups of N neighbouring elements:
// element (i * 32 + lane) * N + j of its head.
template <typename TA, int N, int NI, int KT>
__global__ void __launch_bounds__(128)
attn_conv_prep_kernel(const ConvPrepArgs a) {
    const int lane = threadIdx.x & 31;
    const int head = blockIdx.y * 4 + (threadIdx.x >> 5);
    const int n_heads = a.Hq + (a.own_kv ? 2 * a.Hkv : 0);
    if (head >= n_heads) return;
    const int K = KT > 0 ? KT : a.K;
    const bool is_q = head < a.Hq, is_k = !is_q && head < a.Hq + a.Hkv;
    const int hk = is_q ? head : is_k ? head - a.Hq : head - a.Hq - a.Hkv;
    const int len = (is_q || is_k) ? a.dim : a.vdim;
    const int c0 = is_q ? hk * a.dim : is_k ? a.Hq * a.dim + hk * a.dim : (a.Hq + a.Hkv) * a.dim + hk * a.vdim;
    const int channels = a.own_kv ? (a.Hq + a.Hkv) * a.dim + a.Hkv * a.vdim : a.Hq * a.dim;
    bool on[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) on[i] = (i * 32 + lane) * N < len;
    float w[KT > 0 ? KT : 1][NI][N];
    if (KT > 0) {                                          // the filters are weights: read before the kernel before has ended
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int j = 0; j < N; ++j)
#pragma unroll
                for (int s = 0; s < KT; ++s)
                    w[s][i][j] = on[i] ? load_as_f32(a.taps, a.taps_dtype, (size_t)(c0 + (i * 32 + lane) * N + j) * K + s) : 0.f;
    }
    pdl_wait();
    const TA* proj = (const TA*)a.proj + c0;
    auto run_start = [&](int i) {
        const int t = i * a.run;
        if (t >= a.T) return a.T;
        const int seg = a.tok_seg[t], first = a.cu_q[seg];
        return (t > first && t - first < K - 1) ? min(first + K - 1, a.cu_q[seg + 1]) : t;
    };
    const int t0 = run_start(blockIdx.x), t1 = run_start(blockIdx.x + 1);
    if (t0 >= t1) return;

    float win[KT > 1 ? KT - 1 : 1][NI][N];                 // the last K - 1 inputs, oldest first
    int seg = -1, seg_first = 0, seg_end = 0;
    float* kept = nullptr;
    for (int t = t0; t < t1; ++t) {
        if (t >= seg_end) {
            seg = a.tok_seg[t];
            seg_first = a.cu_q[seg];
            seg_end = a.cu_q[seg + 1];
            kept = a.kept ? a.kept + (long long)a.seg_slot[seg] * a.kept_stride + a.kept_off + c0 : nullptr;
            if (KT > 1) {
#pragma unroll
                for (int s = 0; s < KT - 1; ++s) {
                    const int back = KT - 1 - s;           // t > seg_first: then t is at least K - 1 tokens into its segment
#pragma unroll
                    for (int i = 0; i < NI; ++i) {
#pragma unroll
                        for (int j = 0; j < N; ++j) win[s][i][j] = 0.f;
                        if (!on[i]) continue;
                        const int e = (i * 32 + lane) * N;
                        if (t > seg_first) {
                            ld_vec<TA, N>(proj + (size_t)(t - back) * a.ld + e, win[s][i]);
                        } else {
#pragma unroll
                            for (int j = 0; j < N; ++j) win[s][i][j] = kept[(size_t)s * channels + e + j];
                        }
                    }
                }
            }
        }
        float y[NI][N];
        if (KT > 0) {
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                float u[N];
#pragma unroll
                for (int j = 0; j < N; ++j) u[j] = 0.f;
                if (on[i]) ld_vec<TA, N>(proj + (size_t)t * a.ld + (i * 32 + lane) * N, u);
#pragma unroll
                for (int j = 0; j < N; ++j) {
                    float acc = 0.f;
#pragma unroll
                    for (int s = 0; s < KT - 1; ++s) acc = fmaf(w[s][i][j], win[s][i][j], acc);
                    y[i][j] = fmaf(w[KT - 1][i][j], u[j], acc);
#pragma unroll
                    for (int s = 0; s + 2 < KT; ++s) win[s][i][j] = win[s + 1][i][j];
                    if (KT > 1) win[KT > 1 ? KT - 2 : 0][i][j] = u[j];
                }
            }
        } else {
            const int l = t - seg_first;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int j = 0; j < N; ++j) y[i][j] = 0.f;
                if (!on[i]) continue;
                const int e = (i * 32 + lane) * N;
                for (int back = K - 1; back >= 0; --back) {
                    float u[N];
                    if (back <= l) {
                        ld_vec<TA, N>(proj + (size_t)(t - back) * a.ld + e, u);
                    } else {
#pragma unroll
                        for (int j = 0; j < N; ++j) u[j] = kept[(size_t)(K - 1 - (back - l)) * channels + e + j];
                    }
#pragma unroll
                    for (int j = 0; j < N; ++j)
                        y[i][j] = fmaf(load_as_f32(a.taps, a.taps_dtype, (size_t)(c0 + e + j) * K + (K - 1 - back)), u[j], y[i][j]);
                }
            }
        }
        const int p = a.pos[t];
        float f = 1.f;
        if (a.normed && (is_q || is_k)) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j < N; ++j) ss = fmaf(y[i][j], y[i][j], ss);
            f = 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
        }
        if (is_q && a.temp_every > 0) f *= 1.0f + a.temp_coef * logf((float)((p + 1) / a.temp_every + 1));
        TA* dst = nullptr;
        if (is_q) {
            dst = (TA*)a.q_out + ((size_t)t * a.Hq + hk) * a.D;
        } else if (a.write_kv) {
            const int page = a.block_table[(size_t)seg * a.bt_stride + p / a.page_size];
            if (page >= 0)                                 // a padding row of a captured step has no page
                dst = (TA*)(is_k ? a.kpool : a.vpool) + (((size_t)page * a.Hkv + hk) * a.page_size + p % a.page_size) * a.D;
        }
        if (dst != nullptr) {
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int e = (i * 32 + lane) * N;
                if (e >= a.D) continue;
                float o[N];
#pragma unroll
                for (int j = 0; j < N; ++j) o[j] = on[i] ? y[i][j] * f : 0.f;
                st_vec<TA, N>(dst + e, o);
            }
        }
        // The warp that had the segment's first token renews what the request kept once it has no more use for it: behind
        // the tokens that reach back before the segment.  Row m only needs rows behind m, so they go in order.
        if (K > 1 && t0 <= seg_first && (t == seg_end - 1 || t == seg_first + K - 2)) {
            const int L = seg_end - seg_first;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                if (!on[i]) continue;
                const int e = (i * 32 + lane) * N;
                for (int m = 0; m < K - 1; ++m) {
                    const int back = K - 2 - m;            // tokens before the segment's last one
                    float u[N];
                    if (back < L) {
                        ld_vec<TA, N>(proj + (size_t)(seg_end - 1 - back) * a.ld + e, u);
                    } else {
#pragma unroll
                        for (int j = 0; j < N; ++j) u[j] = kept[(size_t)(m + L) * channels + e + j];
                    }
#pragma unroll
                    for (int j = 0; j < N; ++j) kept[(size_t)m * channels + e + j] = u[j];
                }
            }
        }
    }
}

template <typename TA, int N, int NI>
static int launch_conv_prep(const ConvPrepArgs& a, dim3 grid, cudaStream_t st) {
    switch (a.K) {
        case 1: return rb_launch_pdl(attn_conv_prep_kernel<TA, N, NI, 1>, grid, dim3(128), 0, st, a);
        case 2: return rb_launch_pdl(attn_conv_prep_kernel<TA, N, NI, 2>, grid, dim3(128), 0, st, a);
        case 3: return rb_launch_pdl(attn_conv_prep_kernel<TA, N, NI, 3>, grid, dim3(128), 0, st, a);
        case 4: return rb_launch_pdl(attn_conv_prep_kernel<TA, N, NI, 4>, grid, dim3(128), 0, st, a);
    }
    return rb_launch_pdl(attn_conv_prep_kernel<TA, N, NI, 0>, grid, dim3(128), 0, st, a);
}

RB_EXPORT int rb_attn_conv_prep(const void* proj, int ld, const void* taps, int taps_dtype, int K, float* kept,
                                long long kept_stride, int kept_off, const int* pos, const int* tok_seg, const int* cu_q,
                                const int* seg_slot, const int* block_table, int bt_stride, int page_size, void* kpool,
                                void* vpool, void* q_out, int act_dtype, int T, int Hq, int Hkv, int dim, int vdim, int D,
                                int own_kv, int write_kv, int normed, float eps, float temp_coef, int temp_every, cudaStream_t st) {
    if (T <= 0) return 0;
    if (K < 1 || dim > D || vdim > D || D > 256 || Hq < 1 || Hkv < 1 || (write_kv && !own_kv) || (K > 1 && kept == nullptr))
        return (int)cudaErrorInvalidValue;
    ConvPrepArgs a;
    a.proj = proj; a.ld = ld; a.taps = taps; a.taps_dtype = taps_dtype; a.K = K;
    a.kept = kept; a.kept_stride = kept_stride; a.kept_off = kept_off;
    a.pos = pos; a.tok_seg = tok_seg; a.cu_q = cu_q; a.seg_slot = seg_slot;
    a.block_table = block_table; a.bt_stride = bt_stride; a.page_size = page_size;
    a.kpool = kpool; a.vpool = vpool; a.q_out = q_out;
    a.T = T; a.Hq = Hq; a.Hkv = Hkv; a.dim = dim; a.vdim = vdim; a.D = D;
    a.own_kv = own_kv; a.write_kv = write_kv; a.normed = normed; a.eps = eps; a.temp_coef = temp_coef; a.temp_every = temp_every;
    const int heads = Hq + (own_kv ? 2 * Hkv : 0), head_ctas = (heads + 3) / 4;
    a.run = 1;
    while (a.run < 16 && (long long)(T / (2 * a.run)) * head_ctas >= 148 * 8) a.run *= 2;
    dim3 grid((T + a.run - 1) / a.run, head_ctas);
    const int n = D <= 64 ? 2 : D <= 128 ? 4 : 8;          // neighbouring elements of a lane in bfloat16
    const uintptr_t mask = 2 * n - 1;
    auto al = [&](const void* p) { return p == nullptr || ((uintptr_t)p & mask) == 0; };
    const bool vec = act_dtype == RB_BF16 && dim % n == 0 && vdim % n == 0 && D % n == 0 && ld % n == 0 && al(proj) && al(q_out) &&
                     al(kpool) && al(vpool);
    if (vec && n == 2) return launch_conv_prep<bf16, 2, 1>(a, grid, st);
    if (vec && n == 4) return launch_conv_prep<bf16, 4, 1>(a, grid, st);
    if (vec) return launch_conv_prep<bf16, 8, 1>(a, grid, st);
    // any sizes: single elements, as many groups of 32 as the head has
    if (act_dtype == RB_F32) {
        if (D <= 64) return launch_conv_prep<float, 1, 2>(a, grid, st);
        if (D <= 128) return launch_conv_prep<float, 1, 4>(a, grid, st);
        return launch_conv_prep<float, 1, 8>(a, grid, st);
    }
    if (D <= 64) return launch_conv_prep<bf16, 1, 2>(a, grid, st);
    if (D <= 128) return launch_conv_prep<bf16, 1, 4>(a, grid, st);
    return launch_conv_prep<bf16, 1, 8>(a, grid, st);
}
