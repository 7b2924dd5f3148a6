// What lies between two layers, in one pass over a token's row (float32 throughout, one rounding at the end):
//
//   v  = x[row] + scale * (a[row] + b[row])                 the results the layer before still has to add
//        b may be given undone, as a routed feed-forward leaves it: b = sum_k y[slot_of[row, k]] (+ sigmoid(z[row]) extra[row])
//   x' = v,  or with a history of n earlier streams         x' = sum_(j < n) c_j X_j[row] + c_n v;   X_n[row] <- v
//   out_i = x' * inv(part of the row) * w_i,  i = 1, 2      RMS norms over `groups` equal neighbouring parts of the row
//
// Every piece is optional: no pending results, no history, no norm or one or two of them (they share eps and groups: the
// norms of two sublayers that read the same stream).  x' is written to x_out if that is given (x itself is allowed).
// row = row_idx ? row_idx[r] : r; with row_idx nothing but the norms is written (a row may be listed twice).
#include "common.cuh"

template <typename T> struct StreamParams {
    const float* x;
    float* x_out;
    const int* row_idx;
    const T* a;
    const T* b;
    const T* y;               // a routed feed-forward's expert outputs by slot, or null
    const int* slot_of;       // [rows, top]
    const T* extra;           // what every token takes beside its experts, or null
    const float* extra_z;     // a number a token whose sigmoid multiplies `extra`, or null
    int64_t ld_z;
    int top;
    float scale;
    const float* hist;        // X_0 .. X_(n-1), each [rows, H], hist_stride apart
    float* hist_out;          // X_n, or null
    int64_t hist_stride;
    const float* coef;        // [n + 1], or null: no history
    int n_hist;
    const float* w1;
    const float* w2;
    T* out1;
    T* out2;
    int H, groups;
    float eps;
};

__device__ __forceinline__ float sn_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// H / groups a multiple of 128: a warp's 32 vectors of four lie in one part, so a part's sum of squares is the sum
// of its chunks of 128; a thread's NV vectors stay in registers from the first read to the last write.
// Loads have no condition between them (threads beyond the row read its last vector again): they are in flight together.
template <typename T, int NV>
__global__ void stream_norm_vec_kernel(const StreamParams<T> p) {
    __shared__ float chunk_ss[512];                     // H / 128 chunks
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x;
    const int64_t row = p.row_idx ? p.row_idx[r] : r;
    const bool writes = p.row_idx == nullptr;
    const int n4 = p.H >> 2;
    int at[NV];                                         // this thread's elements
    bool in[NV];
    float4 v[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        in[k] = i < n4;
        at[k] = 4 * min(i, n4 - 1);
        v[k] = *reinterpret_cast<const float4*>(p.x + row * p.H + at[k]);
    }
    if (p.a || p.b || p.y) {
        float gate = 1.f;
        if (p.extra && p.extra_z) gate = sn_sigmoid(p.extra_z[row * p.ld_z]);
        float4 d[NV];
#pragma unroll
        for (int k = 0; k < NV; ++k) d[k] = p.a ? Vec4<T>::load(p.a + row * p.H + at[k]) : make_float4(0.f, 0.f, 0.f, 0.f);
        auto add = [&](const T* src, float f) {
            float4 e[NV];
#pragma unroll
            for (int k = 0; k < NV; ++k) e[k] = Vec4<T>::load(src + at[k]);
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                d[k].x = fmaf(f, e[k].x, d[k].x); d[k].y = fmaf(f, e[k].y, d[k].y);
                d[k].z = fmaf(f, e[k].z, d[k].z); d[k].w = fmaf(f, e[k].w, d[k].w);
            }
        };
        if (p.b) add(p.b + row * p.H, 1.f);
        if (p.y) {
#pragma unroll 2
            for (int c = 0; c < p.top; ++c) add(p.y + (int64_t)p.slot_of[row * p.top + c] * p.H, 1.f);
            if (p.extra) add(p.extra + row * p.H, gate);
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            v[k].x = fmaf(p.scale, d[k].x, v[k].x); v[k].y = fmaf(p.scale, d[k].y, v[k].y);
            v[k].z = fmaf(p.scale, d[k].z, v[k].z); v[k].w = fmaf(p.scale, d[k].w, v[k].w);
        }
    }
    if (p.coef) {
        const float cn = p.coef[p.n_hist];
        float4 acc[NV];
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            if (in[k] && writes && p.hist_out) *reinterpret_cast<float4*>(p.hist_out + row * p.H + at[k]) = v[k];
            acc[k] = make_float4(cn * v[k].x, cn * v[k].y, cn * v[k].z, cn * v[k].w);
        }
        const float* h = p.hist + row * p.H;
        constexpr int AHEAD = NV >= 4 ? 2 : 4;
        for (int j = 0; j < p.n_hist; j += AHEAD) {
            float4 e[AHEAD][NV];
            float c[AHEAD];
#pragma unroll
            for (int q = 0; q < AHEAD; ++q) {
                const int jj = min(j + q, p.n_hist - 1);
                c[q] = j + q < p.n_hist ? p.coef[jj] : 0.f;
#pragma unroll
                for (int k = 0; k < NV; ++k) e[q][k] = *reinterpret_cast<const float4*>(h + jj * p.hist_stride + at[k]);
            }
#pragma unroll
            for (int q = 0; q < AHEAD; ++q) {
                if (j + q >= p.n_hist) break;
#pragma unroll
                for (int k = 0; k < NV; ++k) {
                    acc[k].x = fmaf(c[q], e[q][k].x, acc[k].x); acc[k].y = fmaf(c[q], e[q][k].y, acc[k].y);
                    acc[k].z = fmaf(c[q], e[q][k].z, acc[k].z); acc[k].w = fmaf(c[q], e[q][k].w, acc[k].w);
                }
            }
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) v[k] = acc[k];
    }
    if (writes && p.x_out) {
#pragma unroll
        for (int k = 0; k < NV; ++k)
            if (in[k]) *reinterpret_cast<float4*>(p.x_out + row * p.H + at[k]) = v[k];
    }
    if (!p.out1) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int chunks = p.H >> 7, per = chunks / p.groups;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const float ss = warp_sum(v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w);
        const int c = k * nwarps + warp;
        if (lane == 0 && c < chunks) chunk_ss[c] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = k * nwarps + warp;
        if (c >= chunks) break;
        const int first = c / per * per;
        float ss = 0.f;
        for (int q = lane; q < per; q += 32) ss += chunk_ss[first + q];
        const float inv = rsqrtf(warp_sum(ss) / (float)(p.H / p.groups) + p.eps);
        const float4 n = make_float4(v[k].x * inv, v[k].y * inv, v[k].z * inv, v[k].w * inv);
        const float4 w = *reinterpret_cast<const float4*>(p.w1 + at[k]);
        Vec4<T>::store(p.out1 + (int64_t)r * p.H + at[k], make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
        if (p.out2) {
            const float4 u = *reinterpret_cast<const float4*>(p.w2 + at[k]);
            Vec4<T>::store(p.out2 + (int64_t)r * p.H + at[k], make_float4(n.x * u.x, n.y * u.y, n.z * u.z, n.w * u.w));
        }
    }
}

// Any width and any part size: the row waits in shared memory, a warp a part for the sums of squares.
template <typename T>
__global__ void stream_norm_kernel(const StreamParams<T> p) {
    extern __shared__ float srow[];                     // [H] the row, then [groups] the parts' factors
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x;
    const int64_t row = p.row_idx ? p.row_idx[r] : r;
    const bool writes = p.row_idx == nullptr;
    float* inv_s = srow + p.H;
    float gate = 1.f;
    if (p.extra && p.extra_z) gate = sn_sigmoid(p.extra_z[row * p.ld_z]);
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) {
        const int64_t at = row * p.H + i;
        float d = 0.f;
        if (p.a) d = to_float(p.a[at]);
        if (p.b) d += to_float(p.b[at]);
        if (p.y) {
            float s = 0.f;
            for (int c = 0; c < p.top; ++c) s += to_float(p.y[(int64_t)p.slot_of[row * p.top + c] * p.H + i]);
            if (p.extra) s = fmaf(gate, to_float(p.extra[at]), s);
            d += s;
        }
        float v = fmaf(p.scale, d, p.x[at]);
        if (p.coef) {
            if (writes && p.hist_out) p.hist_out[at] = v;
            v *= p.coef[p.n_hist];
            for (int j = 0; j < p.n_hist; ++j) v = fmaf(p.coef[j], p.hist[j * p.hist_stride + at], v);
        }
        if (writes && p.x_out) p.x_out[at] = v;
        srow[i] = v;
    }
    if (!p.out1) return;
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int part = p.H / p.groups;
    for (int g = warp; g < p.groups; g += nwarps) {
        float ss = 0.f;
        for (int i = lane; i < part; i += 32) ss += srow[g * part + i] * srow[g * part + i];
        ss = warp_sum(ss);
        if (lane == 0) inv_s[g] = rsqrtf(ss / (float)part + p.eps);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.H; i += blockDim.x) {
        const float n = srow[i] * inv_s[i / part];
        p.out1[(int64_t)r * p.H + i] = from_float<T>(n * p.w1[i]);
        if (p.out2) p.out2[(int64_t)r * p.H + i] = from_float<T>(n * p.w2[i]);
    }
}

template <typename T> static int launch_stream_norm(const StreamParams<T>& p, int rows, cudaStream_t stream) {
    const uintptr_t all = (uintptr_t)p.x | (uintptr_t)p.x_out | (uintptr_t)p.a | (uintptr_t)p.b | (uintptr_t)p.y |
                          (uintptr_t)p.extra | (uintptr_t)p.hist | (uintptr_t)p.hist_out | (uintptr_t)p.w1 |
                          (uintptr_t)p.w2 | (uintptr_t)p.out1 | (uintptr_t)p.out2;
    const int part = p.H / p.groups;
    if (part % 128 == 0 && (all & 15) == 0 && p.hist_stride % 4 == 0 && p.H <= 16384) {
        const int n4 = p.H / 4;                          // a multiple of 32
        const int most = rows <= 148 ? 512 : 256;        // few rows: more threads a row; many: more rows at a time
        const int threads = n4 < most ? n4 : (n4 > 8 * most ? 512 : most);
        const int nv = (n4 + threads - 1) / threads;
        if (nv <= 1) return acorn_launch(stream_norm_vec_kernel<T, 1>, dim3(rows), dim3(threads), 0, stream, p);
        if (nv <= 2) return acorn_launch(stream_norm_vec_kernel<T, 2>, dim3(rows), dim3(threads), 0, stream, p);
        if (nv <= 4) return acorn_launch(stream_norm_vec_kernel<T, 4>, dim3(rows), dim3(threads), 0, stream, p);
        if (nv <= 8) return acorn_launch(stream_norm_vec_kernel<T, 8>, dim3(rows), dim3(threads), 0, stream, p);
    }
    const size_t smem = ((size_t)p.H + p.groups) * sizeof(float);
    if (smem > 48 * 1024) return ACORN_ERR_UNSUPPORTED;
    const int threads = p.H >= 2048 ? 512 : (p.H >= 512 ? 256 : 128);
    return acorn_launch(stream_norm_kernel<T>, dim3(rows), dim3(threads), smem, stream, p);
}

extern "C" int acorn_stream_norm(const float* x, float* x_out, const int* row_idx, const void* a, const void* b, const void* y,
                                 const int* slot_of, int top, const void* extra, const float* extra_z, int64_t ld_z,
                                 float scale, const float* hist, int64_t hist_stride, int n_hist, float* hist_out,
                                 const float* coef, const float* w1, void* out1, const float* w2, void* out2, int rows, int H,
                                 int groups, float eps, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (H < 1 || groups < 1 || H % groups || (out1 && !w1) || (out2 && (!w2 || !out1)) || (y && (!slot_of || top < 1)) ||
        (coef && n_hist > 0 && !hist))
        return ACORN_ERR_UNSUPPORTED;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        StreamParams<T> p;
        p.x = x; p.x_out = x_out; p.row_idx = row_idx; p.a = (const T*)a; p.b = (const T*)b; p.y = (const T*)y;
        p.slot_of = slot_of; p.top = top; p.extra = (const T*)extra; p.extra_z = extra_z; p.ld_z = ld_z; p.scale = scale;
        p.hist = hist; p.hist_stride = hist_stride; p.n_hist = n_hist; p.hist_out = hist_out; p.coef = coef;
        p.w1 = w1; p.out1 = (T*)out1; p.w2 = w2; p.out2 = (T*)out2; p.H = H; p.groups = groups; p.eps = eps;
        return launch_stream_norm<T>(p, rows, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
