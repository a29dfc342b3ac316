// The joint between two sublayers of a layer whose norms are elementwise squashes, y = tanh(alpha x) * w + b, with an
// optional blend of every normed row with the row before it.
//
// One kernel does all of it for a float32 residual stream:
//   x[t] = x_in[t] + post(y[t])                     y: the sublayer's output; post: a squash with its own alpha, w, b (a
//                                                   factor per column folded into w and b), or y as it is
//   h[t] = tanh(alpha x[t]) * w + b                 what the next sublayer reads
//   out[t] = h[t] + (h[t - 1] - h[t]) * mu          with a blend vector mu; without one out = h
// Nothing here sums over a row, so a thread owns a few columns and walks a run of neighbouring tokens with h[t - 1] in
// registers.  At the start of a run inside a segment it works h[t - 1] out again from x_in and y (which this launch does
// not change: with a blend x_out is another buffer than x_in).  Before a segment's first token stands what the request
// kept from its last step (zero for a new request); the thread that reads it is also the one that leaves the segment's
// last h there, worked out from the last token's row, so no other launch is needed and no thread reads what another
// has replaced.
// With `rows` the kernel takes the listed rows of x_in only and leaves the stream alone.
#include "common.cuh"

struct SquashVectors { const float* alpha; const float* w; const float* b; };      // alpha: one number

struct JointArgs {
    const float* x_in; float* x_out;                     // x_out null: the stream is not written
    const void* y; int y_f32;                            // null: nothing is added
    SquashVectors post, next;                            // alpha null: absent
    const float* mu;                                     // null: no blend
    float* kept; long long kept_stride; int kept_off;    // a request's last h: row of its slot, from kept_off
    const int* tok_seg; const int* cu_q; const int* seg_slot; const int* rows;
    void* out;
    int T, H, run;
};

// tanh by the hardware's 2^x and reciprocal: an absolute error of a few 1e-7, for results that are rounded to bfloat16 or
// added to a stream whose other terms were.  The float32 path calls the library's.
template <bool FAST>
__device__ __forceinline__ float squash(float x) {
    if (!FAST) return tanhf(x);
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(x * 2.8853900817779268f));
    return 1.0f - __fdividef(2.0f, e + 1.0f);
}

template <int N>
__device__ __forceinline__ void ld_f32(const float* p, float (&v)[N]) {
    if (N == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1 % N] = f.y; v[2 % N] = f.z; v[3 % N] = f.w;
    } else {
        v[0] = *p;
    }
}
template <int N>
__device__ __forceinline__ void st_f32(float* p, const float (&v)[N]) {
    if (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % N], v[2 % N], v[3 % N]);
    else *p = v[0];
}
template <int N>
__device__ __forceinline__ void ld_any(const void* base, int f32, size_t i, float (&v)[N]) {
    if (f32) { ld_f32<N>((const float*)base + i, v); return; }
    const bf16* p = (const bf16*)base + i;
    if (N == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = a.x; v[1 % N] = a.y; v[2 % N] = b.x; v[3 % N] = b.y;
    } else {
        v[0] = __bfloat162float(*p);
    }
}
template <int N> __device__ __forceinline__ void st_act(float* p, const float (&v)[N]) { st_f32<N>(p, v); }
template <int N> __device__ __forceinline__ void st_act(bf16* p, const float (&v)[N]) {
    if (N == 4) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % N]), b = __floats2bfloat162_rn(v[2 % N], v[3 % N]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
    } else {
        *p = __float2bfloat16_rn(v[0]);
    }
}

template <typename TA, int N, bool FAST>
__global__ void __launch_bounds__(128)
tanh_joint_kernel(const JointArgs a) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * N;
    const bool live = c < a.H;
    // the vectors are weights: nobody writes them, so they are read before the kernel before this one has finished
    float pw[N], pb[N], nw[N], nb[N], mu[N];
    const bool has_y = a.y != nullptr, post = a.post.alpha != nullptr, next = a.next.alpha != nullptr, blend = a.mu != nullptr;
    const float pa = post ? *a.post.alpha : 0.f, na = next ? *a.next.alpha : 0.f;
    if (live && post) { ld_f32<N>(a.post.w + c, pw); ld_f32<N>(a.post.b + c, pb); }
    if (live && next) { ld_f32<N>(a.next.w + c, nw); ld_f32<N>(a.next.b + c, nb); }
    if (live && blend) ld_f32<N>(a.mu + c, mu);
    pdl_wait();
    if (!live) return;

    auto load = [&](int t, float (&x)[N], float (&y)[N]) {
        const size_t at = (size_t)t * a.H + c;
        ld_f32<N>(a.x_in + at, x);
        if (has_y) ld_any<N>(a.y, a.y_f32, at, y);
    };
    auto add = [&](float (&x)[N], const float (&y)[N]) {
        if (!has_y) return;
#pragma unroll
        for (int i = 0; i < N; ++i) x[i] += post ? fmaf(squash<FAST>(pa * y[i]), pw[i], pb[i]) : y[i];
    };
    auto stream_at = [&](int t, float (&x)[N]) {
        float y[N];
        load(t, x, y);
        add(x, y);
    };
    auto normed = [&](const float (&x)[N], float (&h)[N]) {
#pragma unroll
        for (int i = 0; i < N; ++i) h[i] = fmaf(squash<FAST>(na * x[i]), nw[i], nb[i]);
    };

    const int r0 = blockIdx.x * a.run, r1 = min(a.T, r0 + a.run);
    float prev[N], x_next[N], y_next[N];
    bool have_prev = false;
    if (r0 < r1) load(a.rows ? a.rows[r0] : r0, x_next, y_next);
    for (int r = r0; r < r1; ++r) {
        const int t = a.rows ? a.rows[r] : r;
        float x[N], y[N], h[N];
#pragma unroll
        for (int i = 0; i < N; ++i) { x[i] = x_next[i]; y[i] = y_next[i]; }
        if (r + 1 < r1) load(a.rows ? a.rows[r + 1] : r + 1, x_next, y_next);      // on its way while this row is worked on
        add(x, y);
        if (a.x_out) st_f32<N>(a.x_out + (size_t)t * a.H + c, x);
        if (!next) continue;
        normed(x, h);
        if (blend) {
            const int seg = a.tok_seg[t];
            const int first = a.cu_q[seg];
            if (t == first) {
                float* home = a.kept + (long long)a.seg_slot[seg] * a.kept_stride + a.kept_off + c;
                ld_f32<N>(home, prev);
                const int last = a.cu_q[seg + 1] - 1;
                if (last == t) {
                    st_f32<N>(home, h);
                } else {
                    float xl[N], hl[N];
                    stream_at(last, xl);
                    normed(xl, hl);
                    st_f32<N>(home, hl);
                }
            } else if (!have_prev) {
                float xp[N];
                stream_at(t - 1, xp);
                normed(xp, prev);
            }
            float o[N];
#pragma unroll
            for (int i = 0; i < N; ++i) { o[i] = fmaf(prev[i] - h[i], mu[i], h[i]); prev[i] = h[i]; }
            have_prev = true;
            st_act<N>((TA*)a.out + (size_t)r * a.H + c, o);
        } else {
            st_act<N>((TA*)a.out + (size_t)r * a.H + c, h);
        }
    }
}

template <typename TA, bool FAST>
static int launch_joint(JointArgs& a, bool vec, cudaStream_t st) {
    const int n = vec ? 4 : 1;
    const int cols = (a.H + 128 * n - 1) / (128 * n);
    // long steps: runs of tokens a thread, so that the vectors are read once and a row's predecessor is at hand
    a.run = (long long)a.T * cols <= 148 * 16 ? 1 : 8;
    dim3 grid((a.T + a.run - 1) / a.run, cols);
    if (vec) return rb_launch_pdl(tanh_joint_kernel<TA, 4, FAST>, grid, dim3(128), 0, st, a);
    return rb_launch_pdl(tanh_joint_kernel<TA, 1, FAST>, grid, dim3(128), 0, st, a);
}

// n_rows: rows of the launch (tokens, or entries of `rows`).
RB_EXPORT int rb_tanh_joint(const float* x_in, float* x_out, const void* y, int y_f32, const float* post_alpha,
                            const float* post_w, const float* post_b, const float* next_alpha, const float* next_w,
                            const float* next_b, const float* mu, float* kept, long long kept_stride, int kept_off,
                            const int* tok_seg, const int* cu_q, const int* seg_slot, const int* rows, void* out,
                            int act_dtype, int n_rows, int H, cudaStream_t st) {
    if (n_rows <= 0 || H <= 0) return 0;
    if (mu != nullptr && (kept == nullptr || next_alpha == nullptr || rows != nullptr || (y != nullptr && x_out == x_in)))
        return (int)cudaErrorInvalidValue;
    if (next_alpha != nullptr && out == nullptr) return (int)cudaErrorInvalidValue;
    JointArgs a;
    a.x_in = x_in; a.x_out = x_out; a.y = y; a.y_f32 = y_f32;
    a.post = {post_alpha, post_w, post_b};
    a.next = {next_alpha, next_w, next_b};
    a.mu = mu; a.kept = kept; a.kept_stride = kept_stride; a.kept_off = kept_off;
    a.tok_seg = tok_seg; a.cu_q = cu_q; a.seg_slot = seg_slot; a.rows = rows; a.out = out;
    a.T = n_rows; a.H = H; a.run = 1;
    auto al = [](const void* p, unsigned m) { return p == nullptr || ((uintptr_t)p & m) == 0; };
    const bool vec = H % 4 == 0 && al(x_in, 15) && al(x_out, 15) && al(y, y_f32 ? 15 : 7) && al(post_w, 15) && al(post_b, 15) &&
                     al(next_w, 15) && al(next_b, 15) && al(mu, 15) && al(kept, 15) && kept_stride % 4 == 0 && kept_off % 4 == 0 &&
                     al(out, act_dtype == RB_F32 ? 15 : 7);
    if (act_dtype == RB_F32) return launch_joint<float, false>(a, vec, st);
    return launch_joint<bf16, true>(a, vec, st);
}
