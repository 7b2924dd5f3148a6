// Several residual streams between two sublayers, in one pass over a token's rows (float32, one rounding at the end):
//
//   y   = a[row], or a routed feed-forward left undone:  sum_k wts[row, k] y[slot_of[row, k]] (+ extra[row])
//   x'_t = sum_s mix[s, t] x_s[row] + scale * put[t] * y          all streams at once from the old ones (mix is [from, to])
//   u   = sum_t take[t] x'_t                                      what the next sublayer reads (take null: the plain sum)
//   out = u * rsqrt(mean(u^2) + eps) * w
//
// Without a pending result x' = x.  The streams lie x_stride apart; x_stride 0: they are all the same rows (a model's first
// sublayer, whose streams are copies of the token rows).  x' goes to x_out (out_stride apart; x itself is allowed when the
// streams lie apart) unless that is null.  row = row_idx ? row_idx[r] : r; with row_idx nothing but the norm is written.
#include "common.cuh"

#define HYPER_MAX_STREAMS 8

template <typename T> struct HyperParams {
    const float* x;
    int64_t x_stride;
    float* x_out;
    int64_t out_stride;
    const int* row_idx;
    const T* a;
    const T* y;
    const int* slot_of;       // [rows, top]
    const float* wts;         // [rows, top], or null: every choice counts once
    int top;
    const T* extra;           // [rows, H] or null
    const float* mix;         // [n, n]
    const float* put;         // [n]
    float scale;
    const float* take;        // [n] or null
    const float* w;
    float eps;
    T* out;                   // [r, H] or null: no norm
    int H, n;
};

// H a multiple of 4: a thread's NV vectors of every stream stay in registers from the first read to the last write.
// Threads beyond the row read its last vector again, so that the loads have no condition between them.
template <typename T, int N, int NV>
__global__ void __launch_bounds__(NV == 4 ? 256 : 512) hyper_norm_vec_kernel(const HyperParams<T> p) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int n4 = p.H >> 2;
    int at[NV];
    bool in[NV];
    float4 x[N][NV], nw[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        in[k] = i < n4;
        at[k] = 4 * min(i, n4 - 1);
        if (NV <= 2 && p.out) nw[k] = *reinterpret_cast<const float4*>(p.w + at[k]);
    }
    float m[N][N], put[N], take[N];                     // (what the model fixes is fetched before the kernel ahead has finished)
#pragma unroll
    for (int t = 0; t < N; ++t) {
        put[t] = p.a || p.y ? p.scale * p.put[t] : 0.f;
        take[t] = p.take ? p.take[t] : 1.f;
#pragma unroll
        for (int s = 0; s < N; ++s) m[s][t] = p.a || p.y ? p.mix[s * N + t] : 0.f;
    }
    pdl_wait();
    pdl_trigger();
    const int64_t row = p.row_idx ? p.row_idx[r] : r;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
#pragma unroll
        for (int s = 0; s < N; ++s) x[s][k] = *reinterpret_cast<const float4*>(p.x + s * p.x_stride + row * p.H + at[k]);
    }
    if (p.a || p.y) {
        float4 d[NV];
        if (p.a) {
#pragma unroll
            for (int k = 0; k < NV; ++k) d[k] = Vec4<T>::load(p.a + row * p.H + at[k]);
        } else {
#pragma unroll
            for (int k = 0; k < NV; ++k) d[k] = p.extra ? Vec4<T>::load(p.extra + row * p.H + at[k]) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
            for (int c = 0; c < p.top; ++c) {
                const T* src = p.y + (int64_t)p.slot_of[row * p.top + c] * p.H;
                const float f = p.wts ? p.wts[row * p.top + c] : 1.f;
#pragma unroll
                for (int k = 0; k < NV; ++k) {
                    const float4 e = Vec4<T>::load(src + at[k]);
                    d[k].x = fmaf(f, e.x, d[k].x); d[k].y = fmaf(f, e.y, d[k].y);
                    d[k].z = fmaf(f, e.z, d[k].z); d[k].w = fmaf(f, e.w, d[k].w);
                }
            }
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            float4 v[N];
#pragma unroll
            for (int t = 0; t < N; ++t) {
                v[t] = make_float4(put[t] * d[k].x, put[t] * d[k].y, put[t] * d[k].z, put[t] * d[k].w);
#pragma unroll
                for (int s = 0; s < N; ++s) {
                    v[t].x = fmaf(m[s][t], x[s][k].x, v[t].x); v[t].y = fmaf(m[s][t], x[s][k].y, v[t].y);
                    v[t].z = fmaf(m[s][t], x[s][k].z, v[t].z); v[t].w = fmaf(m[s][t], x[s][k].w, v[t].w);
                }
            }
#pragma unroll
            for (int t = 0; t < N; ++t) x[t][k] = v[t];
        }
    }
    if (p.x_out && p.row_idx == nullptr) {
#pragma unroll
        for (int t = 0; t < N; ++t)
#pragma unroll
            for (int k = 0; k < NV; ++k)
                if (in[k]) *reinterpret_cast<float4*>(p.x_out + t * p.out_stride + row * p.H + at[k]) = x[t][k];
    }
    if (!p.out) return;
    float4 u[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        u[k] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int t = 0; t < N; ++t) {
            const float f = take[t];
            u[k].x = fmaf(f, x[t][k].x, u[k].x); u[k].y = fmaf(f, x[t][k].y, u[k].y);
            u[k].z = fmaf(f, x[t][k].z, u[k].z); u[k].w = fmaf(f, x[t][k].w, u[k].w);
        }
        if (in[k]) ss += u[k].x * u[k].x + u[k].y * u[k].y + u[k].z * u[k].z + u[k].w * u[k].w;
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)p.H + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        if (!in[k]) continue;
        const float4 w = NV <= 2 ? nw[k] : *reinterpret_cast<const float4*>(p.w + at[k]);
        Vec4<T>::store(p.out + (int64_t)r * p.H + at[k],
                       make_float4(u[k].x * inv * w.x, u[k].y * inv * w.y, u[k].z * inv * w.z, u[k].w * inv * w.w));
    }
}

// Any width, up to HYPER_MAX_STREAMS streams: what the next sublayer reads waits in shared memory for its norm.
template <typename T>
__global__ void __launch_bounds__(512) hyper_norm_kernel(const HyperParams<T> p) {
    extern __shared__ float urow[];                     // [H]
    __shared__ float scratch[32];
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x;
    const int64_t row = p.row_idx ? p.row_idx[r] : r;
    const bool pending = p.a || p.y;
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) {
        float x[HYPER_MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < HYPER_MAX_STREAMS; ++s) x[s] = s < p.n ? p.x[s * p.x_stride + row * p.H + i] : 0.f;
        float d = 0.f;
        if (p.a) {
            d = to_float(p.a[row * p.H + i]);
        } else if (p.y) {
            if (p.extra) d = to_float(p.extra[row * p.H + i]);
            for (int c = 0; c < p.top; ++c)
                d = fmaf(p.wts ? p.wts[row * p.top + c] : 1.f, to_float(p.y[(int64_t)p.slot_of[row * p.top + c] * p.H + i]), d);
        }
        float u = 0.f;
#pragma unroll
        for (int t = 0; t < HYPER_MAX_STREAMS; ++t) {
            if (t >= p.n) break;
            float v = x[t];
            if (pending) {
                v = p.scale * p.put[t] * d;
#pragma unroll
                for (int s = 0; s < HYPER_MAX_STREAMS; ++s)
                    if (s < p.n) v = fmaf(p.mix[s * p.n + t], x[s], v);
            }
            if (p.x_out && p.row_idx == nullptr) p.x_out[t * p.out_stride + row * p.H + i] = v;
            u = fmaf(p.take ? p.take[t] : 1.f, v, u);
        }
        urow[i] = u;
        ss += u * u;
    }
    if (!p.out) return;
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)p.H + p.eps);
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) p.out[(int64_t)r * p.H + i] = from_float<T>(urow[i] * inv * p.w[i]);
}

template <typename T, int N> static int launch_hyper_vec(const HyperParams<T>& p, int rows, cudaStream_t stream) {
    const int n4 = p.H / 4;
    const int most = rows <= 148 || N >= 3 ? 512 : 256;  // few rows: more threads a row; many: more rows at a time, unless a
                                                         // thread's vectors of all streams would take too many registers
    const int nv = (n4 + most - 1) / most;
    const int per = nv <= 1 ? 1 : (nv <= 2 ? 2 : 4);
    const int threads = ((n4 + per - 1) / per + 31) / 32 * 32;
    if (per == 1) return acorn_launch(hyper_norm_vec_kernel<T, N, 1>, dim3(rows), dim3(threads), 0, stream, p);
    if (per == 2) return acorn_launch(hyper_norm_vec_kernel<T, N, 2>, dim3(rows), dim3(threads), 0, stream, p);
    return acorn_launch(hyper_norm_vec_kernel<T, N, 4>, dim3(rows), dim3(threads), 0, stream, p);
}

template <typename T> static int launch_hyper(const HyperParams<T>& p, int rows, cudaStream_t stream) {
    const uintptr_t all = (uintptr_t)p.x | (uintptr_t)p.x_out | (uintptr_t)p.a | (uintptr_t)p.y | (uintptr_t)p.extra |
                          (uintptr_t)p.w | (uintptr_t)p.out;
    if (p.H % 4 == 0 && (all & 15) == 0 && p.x_stride % 4 == 0 && p.out_stride % 4 == 0 && p.n <= 4 && p.H <= 4096) {
        switch (p.n) {
            case 1: return launch_hyper_vec<T, 1>(p, rows, stream);
            case 2: return launch_hyper_vec<T, 2>(p, rows, stream);
            case 3: return launch_hyper_vec<T, 3>(p, rows, stream);
            default: return launch_hyper_vec<T, 4>(p, rows, stream);
        }
    }
    const size_t smem = (size_t)p.H * sizeof(float);
    if (smem > 48 * 1024) return ACORN_ERR_UNSUPPORTED;
    const int threads = p.H >= 2048 ? 512 : (p.H >= 512 ? 256 : 128);
    return acorn_launch(hyper_norm_kernel<T>, dim3(rows), dim3(threads), smem, stream, p);
}

extern "C" int acorn_hyper_norm(const float* x, int64_t x_stride, float* x_out, int64_t out_stride, const int* row_idx,
                                const void* a, const void* y, const int* slot_of, const float* wts, int top, const void* extra,
                                const float* mix, const float* put, float scale, const float* take, const float* w, float eps,
                                void* out, int rows, int H, int n, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (H < 1 || n < 1 || n > HYPER_MAX_STREAMS || (a && y) || ((a || y) && (!mix || !put)) || (y && (!slot_of || top < 1)) ||
        (out && !w) || (x_out == x && n > 1 && x_stride == 0))
        return ACORN_ERR_UNSUPPORTED;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        HyperParams<T> p;
        p.x = x; p.x_stride = x_stride; p.x_out = x_out; p.out_stride = out_stride; p.row_idx = row_idx;
        p.a = (const T*)a; p.y = (const T*)y; p.slot_of = slot_of; p.wts = wts; p.top = top; p.extra = (const T*)extra;
        p.mix = mix; p.put = put; p.scale = scale; p.take = take; p.w = w; p.eps = eps; p.out = (T*)out; p.H = H; p.n = n;
        return launch_hyper<T>(p, rows, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
