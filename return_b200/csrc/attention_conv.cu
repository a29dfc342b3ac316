// Between an attention's projections and its paged attention kernel, for attentions whose q, k and v pass a short causal
// convolution over time and whose q and k heads are normed one by one:
//   y[t] = sum_j taps[:, j] * u[t - K + 1 + j]      u: the projected row [q | k | v], channel by channel; before a step's
//                                                   first token of a request come the inputs the request kept (zero for a
//                                                   new request)
//   q, k heads: y / sqrt(mean(y^2) + eps)           without a weight; can be left out
//   q heads:    times 1 + coef * ln((p + 1) / every + 1), the quotient without its remainder, p the position
//   q heads to a buffer of heads padded to D with zeros, k and v heads (padded) into the cache's pages.
// Compiled for a filter length, -DCONV_TAPS=1 .. 4 or 0 (any, read at run time), and a size of the padded heads,
// -DHEAD_LANES=64, 128 or 256 (heads of up to so many elements).
//
// A group of lanes owns one head (eight neighbouring elements a lane in bfloat16, so a warp may hold several heads) and
// walks a run of neighbouring tokens of the packed step with the last K - 1 inputs of its channels in registers (K up to
// 4; longer filters read them again).  A run that would begin among the first K - 1 tokens of a segment, but not at its
// first, leaves those tokens to the run before it: so the kept inputs are read by one group, the one that has the
// segment's first token, and that group leaves the segment's last K - 1 inputs in their place.
// The kept inputs of a request: K - 1 rows of [q | k | v] channels, oldest first, float32.
#include "common.cuh"

#if !defined(CONV_TAPS) || !defined(HEAD_LANES)
#error "compile with -DCONV_TAPS=0 .. 4 and -DHEAD_LANES=64, 128 or 256"
#endif
static_assert(CONV_TAPS >= 0 && CONV_TAPS <= 4, "filter lengths held in registers: 1 to 4; 0: any");
static_assert(HEAD_LANES == 64 || HEAD_LANES == 128 || HEAD_LANES == 256, "heads of up to 64, 128 or 256 elements");
constexpr int KT = CONV_TAPS;
constexpr int AHEAD = 4;         // tokens whose inputs are asked for together

struct ConvPrepArgs {
    const void* proj; int ld;
    const float* taps; int K;                              // [K][channels], the last row for the token itself
    float* kept; long long kept_stride; int kept_off;
    const int* pos; const int* tok_seg; const int* cu_q; const int* seg_slot; const int* block_table; int bt_stride, page_size;
    void* kpool; void* vpool; void* q_out;
    int T, Hq, Hkv, dim, vdim, D, own_kv, write_kv, normed;
    float inv_dim, eps, temp_coef; int temp_every;                  // temp_every 0: no temperature
    int run;
};

template <typename TA, int N>
__device__ __forceinline__ void ld_vec(const TA* p, float (&v)[N]);
template <> __device__ __forceinline__ void ld_vec<float, 1>(const float* p, float (&v)[1]) { v[0] = *p; }
template <> __device__ __forceinline__ void ld_vec<bf16, 1>(const bf16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
template <> __device__ __forceinline__ void ld_vec<bf16, 8>(const bf16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
// A lane's elements as they lie in memory: loaded now, converted when their token's turn comes (a conversion right behind
// its load would wait for it there).
template <typename TA, int N> struct Raw { TA x; };
template <> struct Raw<bf16, 8> { uint4 x; };
template <typename TA, int N> __device__ __forceinline__ void cook(const Raw<TA, N>& r, float (&v)[N]) { ld_vec<TA, N>((const TA*)&r.x, v); }

template <typename TA, int N>
__device__ __forceinline__ void st_vec(TA* p, const float (&v)[N]);
template <> __device__ __forceinline__ void st_vec<float, 1>(float* p, const float (&v)[1]) { *p = v[0]; }
template <> __device__ __forceinline__ void st_vec<bf16, 1>(bf16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
template <> __device__ __forceinline__ void st_vec<bf16, 8>(bf16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// LPH lanes a head; a lane holds NI groups of N neighbouring elements: element (i * LPH + lane) * N + j of its head.
template <typename TA, int N, int NI, int LPH>
__global__ void __launch_bounds__(128, 4)
attn_conv_prep_kernel(const ConvPrepArgs a) {
    const int lane = threadIdx.x % LPH;
    const int n_heads = a.Hq + (a.own_kv ? 2 * a.Hkv : 0);
    const int wanted = blockIdx.y * (128 / LPH) + threadIdx.x / LPH;
    const bool active = wanted < n_heads;                  // a group without a head walks the last one's, and writes nothing
    const int head = active ? wanted : n_heads - 1;
    const int K = KT > 0 ? KT : a.K;
    const bool is_q = head < a.Hq, is_k = !is_q && head < a.Hq + a.Hkv;
    const int hk = is_q ? head : is_k ? head - a.Hq : head - a.Hq - a.Hkv;
    const int len = (is_q || is_k) ? a.dim : a.vdim;
    const int c0 = is_q ? hk * a.dim : is_k ? a.Hq * a.dim + hk * a.dim : (a.Hq + a.Hkv) * a.dim + hk * a.vdim;
    const int channels = a.own_kv ? (a.Hq + a.Hkv) * a.dim + a.Hkv * a.vdim : a.Hq * a.dim;
    bool on[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) on[i] = (i * LPH + lane) * N < len;
    float w[KT > 0 ? KT : 1][NI][N];
    if (KT > 0) {                                          // the filters are weights: read before the kernel before has ended
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int s = 0; s < KT; ++s) {
                const float* at = a.taps + (size_t)s * channels + c0 + (on[i] ? (i * LPH + lane) * N : 0);
                if (N == 8) {
                    const float4 x = *reinterpret_cast<const float4*>(at), y = *reinterpret_cast<const float4*>(at + 4);
                    w[s][i][0] = x.x; w[s][i][1 % N] = x.y; w[s][i][2 % N] = x.z; w[s][i][3 % N] = x.w;
                    w[s][i][4 % N] = y.x; w[s][i][5 % N] = y.y; w[s][i][6 % N] = y.z; w[s][i][7 % N] = y.w;
                } else {
                    w[s][i][0] = *at;
                }
            }
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
    int seg = -1, seg_first = 0, seg_end = 0, pos_first = 0;
    int page_first = 0, page_end = -1;                     // positions of the page that dst_page points at
    int temp_end = -1;                                     // the first position with another temperature
    float temp = 1.f;
    TA* dst_page = nullptr;
    float* kept = nullptr;
    Raw<TA, N> ahead[AHEAD][NI];                           // the inputs of the next few tokens, asked for together
    for (int tb = t0; tb < t1; tb += AHEAD) {
#pragma unroll
        for (int n = 0; n < AHEAD; ++n)
#pragma unroll
            for (int i = 0; i < NI; ++i) {                 // a lane or a token without an element reads the head's first
                const bool there = on[i] && tb + n < t1;
                ahead[n][i] = *reinterpret_cast<const Raw<TA, N>*>(proj + (size_t)(there ? tb + n : tb) * a.ld + (there ? (i * LPH + lane) * N : 0));
            }
#pragma unroll
        for (int n = 0; n < AHEAD; ++n) {
            const int t = tb + n;
            if (t >= t1) break;
            if (t >= seg_end) {
                seg = a.tok_seg[t];
                seg_first = a.cu_q[seg];
                seg_end = a.cu_q[seg + 1];
                pos_first = a.pos[seg_first];
                page_end = temp_end = -1;
                kept = a.kept ? a.kept + (long long)a.seg_slot[seg] * a.kept_stride + a.kept_off + c0 : nullptr;
                if (KT > 1) {
#pragma unroll
                    for (int s = 0; s < KT - 1; ++s) {
                        const int back = KT - 1 - s;       // t > seg_first: then t is at least K - 1 tokens into its segment
#pragma unroll
                        for (int i = 0; i < NI; ++i) {
#pragma unroll
                            for (int j = 0; j < N; ++j) win[s][i][j] = 0.f;
                            if (!on[i]) continue;
                            const int e = (i * LPH + lane) * N;
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
            const int p = pos_first + (t - seg_first);
            if (!is_q && a.write_kv && p >= page_end) {
                const int block = p / a.page_size;
                const int page = a.block_table[(size_t)seg * a.bt_stride + block];           // -1: a padding row of a captured step
                page_first = block * a.page_size;
                page_end = page_first + a.page_size;
                dst_page = page < 0 ? nullptr : (TA*)(is_k ? a.kpool : a.vpool) + ((size_t)page * a.Hkv + hk) * a.page_size * a.D;
            }
            if (is_q && a.temp_every > 0 && p >= temp_end) {
                const int runs = (p + 1) / a.temp_every;
                temp = 1.0f + a.temp_coef * logf((float)(runs + 1));
                temp_end = (runs + 1) * a.temp_every - 1;
            }
            float y[NI][N];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                if (KT > 0) {
                    float u[N];
                    cook<TA, N>(ahead[n][i], u);
#pragma unroll
                    for (int j = 0; j < N; ++j) {
                        if (!on[i]) u[j] = 0.f;
                        float acc = 0.f;
#pragma unroll
                        for (int s = 0; s < KT - 1; ++s) acc = fmaf(w[s][i][j], win[s][i][j], acc);
                        y[i][j] = fmaf(w[KT > 0 ? KT - 1 : 0][i][j], u[j], acc);
#pragma unroll
                        for (int s = 0; s + 2 < KT; ++s) win[s][i][j] = win[s + 1][i][j];
                        if (KT > 1) win[KT > 1 ? KT - 2 : 0][i][j] = u[j];
                    }
                } else {
                    const int l = t - seg_first, e = (i * LPH + lane) * N;
#pragma unroll
                    for (int j = 0; j < N; ++j) y[i][j] = 0.f;
                    if (!on[i]) continue;
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
                            y[i][j] = fmaf(a.taps[(size_t)(K - 1 - back) * channels + c0 + e + j], u[j], y[i][j]);
                    }
                }
            }
            float f = 1.f;
            if (a.normed) {                                // every lane takes part in the sum; values are not normed
                float ss = 0.f;
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int j = 0; j < N; ++j) ss = fmaf(y[i][j], y[i][j], ss);
#pragma unroll
                for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
                // values that are rounded to bfloat16 take the approximate root (two units in the last place)
                if (is_q || is_k) f = sizeof(TA) == 2 ? rsqrtf(fmaf(ss, a.inv_dim, a.eps)) : 1.0f / sqrtf(ss / (float)a.dim + a.eps);
            }
            f *= temp;
            TA* dst = nullptr;
            if (is_q) dst = (TA*)a.q_out + ((size_t)t * a.Hq + hk) * a.D;
            else if (a.write_kv && dst_page != nullptr) dst = dst_page + (p - page_first) * a.D;
            if (active && dst != nullptr) {
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int e = (i * LPH + lane) * N;
                    if (e >= a.D) continue;
                    float o[N];
#pragma unroll
                    for (int j = 0; j < N; ++j) o[j] = on[i] ? y[i][j] * f : 0.f;
                    st_vec<TA, N>(dst + e, o);
                }
            }
            // The warp that had the segment's first token renews what the request kept once it has no more use for it:
            // behind the tokens that reach back before the segment.  Row m only needs rows behind m, so they go in order.
            if (K > 1 && active && t0 <= seg_first && (t == seg_end - 1 || t == seg_first + K - 2)) {
                const int L = seg_end - seg_first;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    if (!on[i]) continue;
                    const int e = (i * LPH + lane) * N;
                    for (int m = 0; m < K - 1; ++m) {
                        const int back = K - 2 - m;        // tokens before the segment's last one
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
}

RB_EXPORT int rb_attn_conv_prep(const void* proj, int ld, const float* taps, int K, float* kept,
                                long long kept_stride, int kept_off, const int* pos, const int* tok_seg, const int* cu_q,
                                const int* seg_slot, const int* block_table, int bt_stride, int page_size, void* kpool,
                                void* vpool, void* q_out, int act_dtype, int T, int Hq, int Hkv, int dim, int vdim, int D,
                                int own_kv, int write_kv, int normed, float eps, float temp_coef, int temp_every, cudaStream_t st) {
    if (T <= 0) return 0;
    if (K < 1 || (KT > 0 && K != KT) || dim > D || vdim > D || D > HEAD_LANES || Hq < 1 || Hkv < 1 || (write_kv && !own_kv) || (K > 1 && kept == nullptr))
        return (int)cudaErrorInvalidValue;
    ConvPrepArgs a;
    a.proj = proj; a.ld = ld; a.taps = taps; a.K = K;
    a.kept = kept; a.kept_stride = kept_stride; a.kept_off = kept_off;
    a.pos = pos; a.tok_seg = tok_seg; a.cu_q = cu_q; a.seg_slot = seg_slot;
    a.block_table = block_table; a.bt_stride = bt_stride; a.page_size = page_size;
    a.kpool = kpool; a.vpool = vpool; a.q_out = q_out;
    a.T = T; a.Hq = Hq; a.Hkv = Hkv; a.dim = dim; a.vdim = vdim; a.D = D;
    a.own_kv = own_kv; a.write_kv = write_kv; a.normed = normed; a.inv_dim = 1.0f / (float)dim; a.eps = eps; a.temp_coef = temp_coef; a.temp_every = temp_every;
    const int heads = Hq + (own_kv ? 2 * Hkv : 0);
    auto al = [&](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = act_dtype == RB_BF16 && dim % 8 == 0 && vdim % 8 == 0 && D % 8 == 0 && ld % 8 == 0 && al(proj) && al(q_out) && al(taps) &&
                     al(kpool) && al(vpool);
    constexpr int LPH = HEAD_LANES / 8;                    // lanes of a head when each holds eight neighbouring elements
    const int head_ctas = vec ? (heads + 128 / LPH - 1) / (128 / LPH) : (heads + 3) / 4;
    // runs just long enough that one wave of CTAs (four an SM) covers the step; very long steps take several waves
    const long long slots = 4LL * rb_num_sms();
    a.run = slots > 0 ? (int)(((long long)T * head_ctas + slots - 1) / slots) : 16;
    if (a.run > 2) a.run = (a.run + AHEAD - 1) / AHEAD * AHEAD;
    if (a.run > 64) a.run = 64;
    dim3 grid((T + a.run - 1) / a.run, head_ctas);
    if (vec) return rb_launch_pdl(attn_conv_prep_kernel<bf16, 8, 1, LPH>, grid, dim3(128), 0, st, a);
    // any sizes: single elements, as many groups of 32 as the head has
    if (act_dtype == RB_F32) return rb_launch_pdl(attn_conv_prep_kernel<float, 1, HEAD_LANES / 32, 32>, grid, dim3(128), 0, st, a);
    return rb_launch_pdl(attn_conv_prep_kernel<bf16, 1, HEAD_LANES / 32, 32>, grid, dim3(128), 0, st, a);
}
