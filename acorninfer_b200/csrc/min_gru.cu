// A gated recurrence whose gates read the current token only (minGRU), over every row's tokens, channel by channel:
//
//   z = sigmoid(proj_z + b_z),   u = proj_u + b_u,   c = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S <- (1 - z) S + z c                             float32, in the request's state slot between steps
//   out = S * silu(proj_g)
//
// proj holds [z | u | g] of `width` columns each, as projected.  A thread takes V neighbouring channels.  Rows of a few
// tokens run in one piece (min_gru_rows); long rows in segments side by side, in two passes: the first gives every segment
// its product of (1 - z) and its state from zero (the row's own state stands in front of them), the second folds those
// of the segments before its own and walks its tokens again.
#include "common.cuh"

template <typename T> struct GruParams {
    const T* proj;            // [T, ld]
    int64_t ld;
    const float* bias;        // [2 width]: of z, then of u
    float* state;             // [slots, slot_stride] float32, this layer's part from state_off on
    int64_t slot_stride, state_off;
    const int* row_start;
    const int* row_slot;
    T* out;                   // [T, width]
    int width;
    float* seg_a;             // [rows, nseg, width] product of (1 - z) over a segment
    float* seg_b;             // [rows, nseg + 1, width] entry 0: the row's state before the step; s + 1: segment s from zero
    int seg_tokens, nseg;
};

template <typename T> __device__ __forceinline__ float gru_sigmoid(float x);
template <> __device__ __forceinline__ float gru_sigmoid<float>(float x) { return 1.f / (1.f + expf(-x)); }
// under bfloat16 projections: the fast float32 instructions (relative error about 2^-21)
template <> __device__ __forceinline__ float gru_sigmoid<bf16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <typename T, int V> struct Lanes;
template <typename T> struct Lanes<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_float(*p); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_float<T>(v[0]); }
};
template <typename T> struct Lanes<T, 4> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[4]) {
        const float4 x = Vec4<T>::load(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(T* p, const float (&v)[4]) {
        Vec4<T>::store(p, make_float4(v[0], v[1], v[2], v[3]));
    }
};

// the gate and the candidate of a token's channel
template <typename T>
__device__ __forceinline__ void gru_gates(float z_in, float u, float& z, float& c) {
    z = gru_sigmoid<T>(z_in);
    c = u >= 0.f ? u + 0.5f : gru_sigmoid<T>(u);
}

#define GRU_AHEAD 4           // tokens whose loads are in flight together

// tokens t0 .. t1-1: S on, outputs written
template <typename T, int V>
__device__ __forceinline__ void gru_walk(const GruParams<T>& p, int c0, int64_t t0, int64_t t1, const float (&bz)[V],
                                         const float (&bu)[V], float (&S)[V]) {
    for (int64_t t = t0; t < t1; t += GRU_AHEAD) {
        float z[GRU_AHEAD][V], u[GRU_AHEAD][V], g[GRU_AHEAD][V];
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k) {
            if (t + k < t1) {
                const T* row = p.proj + (t + k) * p.ld + c0;
                Lanes<T, V>::load(row, z[k]);
                Lanes<T, V>::load(row + p.width, u[k]);
                Lanes<T, V>::load(row + 2 * (int64_t)p.width, g[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k) {
            if (t + k < t1) {
                float o[V];
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    float zz, cc;
                    gru_gates<T>(z[k][i] + bz[i], u[k][i] + bu[i], zz, cc);
                    S[i] = fmaf(1.f - zz, S[i], zz * cc);
                    o[i] = S[i] * (g[k][i] * gru_sigmoid<T>(g[k][i]));
                }
                Lanes<T, V>::store(p.out + (t + k) * p.width + c0, o);
            }
        }
    }
}

template <typename T, int V>
__global__ void __launch_bounds__(128) min_gru_rows_kernel(const GruParams<T> p) {
    pdl_wait();
    pdl_trigger();
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * V, r = blockIdx.y;
    if (c0 >= p.width) return;
    float* st = p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0;
    float bz[V], bu[V], S[V];
    Lanes<float, V>::load(p.bias + c0, bz);
    Lanes<float, V>::load(p.bias + p.width + c0, bu);
    Lanes<float, V>::load(st, S);
    gru_walk<T, V>(p, c0, p.row_start[r], p.row_start[r + 1], bz, bu, S);
    Lanes<float, V>::store(st, S);
}

// first pass: blockIdx.y = row * (nseg - 1) + segment (a row's last segment needs none of this)
template <typename T, int V>
__global__ void __launch_bounds__(128) min_gru_segments_kernel(const GruParams<T> p) {
    pdl_wait();
    pdl_trigger();
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const int r = blockIdx.y / (p.nseg - 1), s = blockIdx.y % (p.nseg - 1);
    if (c0 >= p.width) return;
    const int64_t first = p.row_start[r], end = p.row_start[r + 1];
    float* sb = p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0;
    if (s == 0) {
        float S[V];
        Lanes<float, V>::load(p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0, S);
        Lanes<float, V>::store(sb, S);
    }
    const int64_t t0 = first + (int64_t)s * p.seg_tokens, t1 = t0 + p.seg_tokens;
    if (t1 >= end) return;                              // the row's last segment, or beyond it
    float bz[V], bu[V], A[V], B[V];
    Lanes<float, V>::load(p.bias + c0, bz);
    Lanes<float, V>::load(p.bias + p.width + c0, bu);
#pragma unroll
    for (int i = 0; i < V; ++i) { A[i] = 1.f; B[i] = 0.f; }
    for (int64_t t = t0; t < t1; t += GRU_AHEAD) {
        float z[GRU_AHEAD][V], u[GRU_AHEAD][V];
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k) {
            if (t + k < t1) {
                const T* row = p.proj + (t + k) * p.ld + c0;
                Lanes<T, V>::load(row, z[k]);
                Lanes<T, V>::load(row + p.width, u[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < GRU_AHEAD; ++k) {
            if (t + k < t1) {
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    float zz, cc;
                    gru_gates<T>(z[k][i] + bz[i], u[k][i] + bu[i], zz, cc);
                    A[i] *= 1.f - zz;
                    B[i] = fmaf(1.f - zz, B[i], zz * cc);
                }
            }
        }
    }
    Lanes<float, V>::store(p.seg_a + ((int64_t)r * p.nseg + s) * p.width + c0, A);
    Lanes<float, V>::store(sb + (int64_t)(s + 1) * p.width, B);
}

// second pass: blockIdx.y = row * nseg + segment
template <typename T, int V>
__global__ void __launch_bounds__(128) min_gru_finish_kernel(const GruParams<T> p) {
    pdl_wait();
    pdl_trigger();
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const int r = blockIdx.y / p.nseg, s = blockIdx.y % p.nseg;
    if (c0 >= p.width) return;
    const int64_t first = p.row_start[r], end = p.row_start[r + 1];
    const int64_t t0 = first + (int64_t)s * p.seg_tokens;
    if (t0 >= end) return;
    const int64_t t1 = min(t0 + (int64_t)p.seg_tokens, end);
    const float* sa = p.seg_a + (int64_t)r * p.nseg * p.width + c0;
    const float* sb = p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0;
    float bz[V], bu[V], S[V];
    Lanes<float, V>::load(p.bias + c0, bz);
    Lanes<float, V>::load(p.bias + p.width + c0, bu);
    Lanes<float, V>::load(sb, S);
#pragma unroll 4
    for (int q = 0; q < s; ++q) {
        float A[V], B[V];
        Lanes<float, V>::load(sa + (int64_t)q * p.width, A);
        Lanes<float, V>::load(sb + (int64_t)(q + 1) * p.width, B);
#pragma unroll
        for (int i = 0; i < V; ++i) S[i] = fmaf(A[i], S[i], B[i]);
    }
    gru_walk<T, V>(p, c0, t0, t1, bz, bu, S);
    if (t1 == end) Lanes<float, V>::store(p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0, S);
}

template <typename T, int V>
static int launch_gru(const GruParams<T>& p, int rows, int pass, cudaStream_t stream) {
    const int lanes = (p.width + V - 1) / V;
    const int threads = lanes >= 128 ? 128 : (lanes + 31) / 32 * 32;
    const int bx = (lanes + threads - 1) / threads;
    if (pass == 0) return acorn_launch(min_gru_rows_kernel<T, V>, dim3(bx, rows), dim3(threads), 0, stream, p);
    if (pass == 1)
        return acorn_launch(min_gru_segments_kernel<T, V>, dim3(bx, rows * (p.nseg - 1)), dim3(threads), 0, stream, p);
    return acorn_launch(min_gru_finish_kernel<T, V>, dim3(bx, rows * p.nseg), dim3(threads), 0, stream, p);
}

// pass 0: rows in one piece; passes 1 and 2: in nseg segments of seg_tokens (seg_a, seg_b as above; nseg >= 2)
extern "C" int acorn_min_gru(const void* proj, int64_t ld, const float* bias, float* state, int64_t slot_stride,
                             int64_t state_off, const int* row_start, const int* row_slot, void* out, int rows, int width,
                             int pass, int seg_tokens, int nseg, float* seg_a, float* seg_b, int dtype, cudaStream_t stream) {
    if (rows <= 0 || width <= 0) return 0;
    if (pass < 0 || pass > 2 || (pass > 0 && (nseg < 2 || seg_tokens < 1 || !seg_a || !seg_b)) ||
        (int64_t)rows * (pass ? nseg : 1) > 65535)
        return ACORN_ERR_UNSUPPORTED;
    const uintptr_t all = (uintptr_t)proj | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)out | (uintptr_t)seg_a | (uintptr_t)seg_b;
    const bool vec = width % 4 == 0 && ld % 4 == 0 && slot_stride % 4 == 0 && state_off % 4 == 0 && (all & 15) == 0;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        GruParams<T> p;
        p.proj = (const T*)proj; p.ld = ld; p.bias = bias; p.state = state; p.slot_stride = slot_stride;
        p.state_off = state_off; p.row_start = row_start; p.row_slot = row_slot; p.out = (T*)out; p.width = width;
        p.seg_a = seg_a; p.seg_b = seg_b; p.seg_tokens = seg_tokens; p.nseg = nseg;
        return vec ? launch_gru<T, 4>(p, rows, pass, stream) : launch_gru<T, 1>(p, rows, pass, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
