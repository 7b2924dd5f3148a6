// A gated recurrence whose gates read the current token only (minGRU), over every row's tokens, channel by channel:
//
//   z = sigmoid(proj_z + b_z),   u = proj_u + b_u,   c = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S <- (1 - z) S + z c                             float32, in the request's state slot between steps
//   out = S * silu(proj_g)
//
// proj holds [z | u | g] of `width` columns each, as projected.  A thread takes V neighbouring channels.  Rows of a few
// tokens: a thread walks its channels (min_gru_rows).  Longer rows: a block takes a segment of GRU_SEG tokens by 32 V
// channels, a warp GRU_WARP_TOKENS of them, whose loads are all in flight at once; a token maps S to a S + b, maps compose, and
// the warps' composed maps meet in shared memory.  Rows of several segments take two passes: the first leaves every
// segment's composed map in memory (the row's own state in front of them), the second composes those of the segments before
// its own, shared out over its warps, and writes the outputs.
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
    float* seg_a;             // [rows, nseg, width] a of a segment's map (the product of its 1 - z)
    float* seg_b;             // [rows, nseg + 1, width] entry 0: the row's state before the step; s + 1: b of segment s's map
    int nseg;
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
template <> struct Lanes<float, 2> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[2]) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        v[0] = x.x; v[1] = x.y;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[2]) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
};
template <> struct Lanes<bf16, 2> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[2]) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        v[0] = x.x; v[1] = x.y;
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[2]) {
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
    }
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

#define GRU_WARP_TOKENS 8
#define GRU_WARPS 16
#define GRU_SEG (GRU_WARP_TOKENS * GRU_WARPS)

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
    const int64_t end = p.row_start[r + 1];
    for (int64_t t = p.row_start[r]; t < end; ++t) {
        const T* row = p.proj + t * p.ld + c0;
        float z[V], u[V], g[V];
        Lanes<T, V>::load(row, z);
        Lanes<T, V>::load(row + p.width, u);
        Lanes<T, V>::load(row + 2 * (int64_t)p.width, g);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            float zz, cc;
            gru_gates<T>(z[i] + bz[i], u[i] + bu[i], zz, cc);
            S[i] = fmaf(1.f - zz, S[i], zz * cc);
            g[i] = S[i] * (g[i] * gru_sigmoid<T>(g[i]));
        }
        Lanes<T, V>::store(p.out + t * p.width + c0, g);
    }
    Lanes<float, V>::store(st, S);
}

// FINISH false: the first pass, blockIdx.y = row * (nseg - 1) + segment (a row's last segment needs none of it);
// FINISH true: the second, blockIdx.y = row * nseg + segment; with nseg = 1 the only one, from the row's state itself.
template <typename T, int V, bool FINISH>
__global__ void __launch_bounds__(32 * GRU_WARPS) min_gru_segment_kernel(const GruParams<T> p) {
    __shared__ __align__(16) float s_a[GRU_WARPS][32 * V], s_b[GRU_WARPS][32 * V];    // the warps' maps of their tokens
    __shared__ __align__(16) float p_a[FINISH ? GRU_WARPS : 1][32 * V], p_b[FINISH ? GRU_WARPS : 1][32 * V];   // of segments before
    pdl_wait();
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per_row = FINISH ? p.nseg : p.nseg - 1;
    const int r = blockIdx.y / per_row, s = blockIdx.y % per_row;
    const int c0 = (blockIdx.x * 32 + lane) * V;
    const bool on = c0 < p.width;
    const int64_t first = p.row_start[r], end = p.row_start[r + 1];
    const int64_t seg0 = first + (int64_t)s * GRU_SEG;
    float* st = p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0;
    if (!FINISH && s == 0 && warp == 0 && on) {
        float S[V];
        Lanes<float, V>::load(st, S);
        Lanes<float, V>::store(p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0, S);
    }
    if (FINISH ? seg0 >= end : seg0 + GRU_SEG >= end) return;        // (the same for the whole block)
    const int64_t t0 = seg0 + warp * GRU_WARP_TOKENS;
    const int n = on ? (int)max((int64_t)0, min((int64_t)GRU_WARP_TOKENS, end - t0)) : 0;
    float a[GRU_WARP_TOKENS][V], b[GRU_WARP_TOKENS][V], g[GRU_WARP_TOKENS][V];
#pragma unroll
    for (int k = 0; k < GRU_WARP_TOKENS; ++k) {
        if (k < n) {
            const T* row = p.proj + (t0 + k) * p.ld + c0;
            Lanes<T, V>::load(row, a[k]);
            Lanes<T, V>::load(row + p.width, b[k]);
            if (FINISH) Lanes<T, V>::load(row + 2 * (int64_t)p.width, g[k]);
        }
    }
    float bz[V], bu[V], A[V], B[V];
#pragma unroll
    for (int i = 0; i < V; ++i) { bz[i] = bu[i] = 0.f; A[i] = 1.f; B[i] = 0.f; }
    if (on) {
        Lanes<float, V>::load(p.bias + c0, bz);
        Lanes<float, V>::load(p.bias + p.width + c0, bu);
    }
    float S[V];
#pragma unroll
    for (int i = 0; i < V; ++i) S[i] = 0.f;
    if (FINISH && on) {
        if (p.nseg == 1) {
            Lanes<float, V>::load(st, S);
        } else {
            Lanes<float, V>::load(p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0, S);
            // this warp's share of the segments before, composed in their order
            const int share = (s + GRU_WARPS - 1) / GRU_WARPS;
            const float* sa = p.seg_a + (int64_t)r * p.nseg * p.width + c0;
            const float* sb = p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0;
            for (int q = warp * share; q < min(s, (warp + 1) * share); ++q) {
                float x[V], y[V];
                Lanes<float, V>::load(sa + (int64_t)q * p.width, x);
                Lanes<float, V>::load(sb + (int64_t)(q + 1) * p.width, y);
#pragma unroll
                for (int i = 0; i < V; ++i) { B[i] = fmaf(x[i], B[i], y[i]); A[i] *= x[i]; }
            }
        }
        Lanes<float, V>::store(&p_a[warp][lane * V], A);
        Lanes<float, V>::store(&p_b[warp][lane * V], B);
#pragma unroll
        for (int i = 0; i < V; ++i) { A[i] = 1.f; B[i] = 0.f; }
    }
#pragma unroll
    for (int k = 0; k < GRU_WARP_TOKENS; ++k) {
        if (k < n) {
#pragma unroll
            for (int i = 0; i < V; ++i) {
                float zz, cc;
                gru_gates<T>(a[k][i] + bz[i], b[k][i] + bu[i], zz, cc);
                a[k][i] = 1.f - zz;
                b[k][i] = zz * cc;
                A[i] *= a[k][i];
                B[i] = fmaf(a[k][i], B[i], b[k][i]);
            }
        }
    }
    Lanes<float, V>::store(&s_a[warp][lane * V], A);
    Lanes<float, V>::store(&s_b[warp][lane * V], B);
    __syncthreads();
    if (!FINISH) {
        if (warp == 0 && on) {
            float X[V], Y[V];
#pragma unroll
            for (int i = 0; i < V; ++i) { X[i] = 1.f; Y[i] = 0.f; }
#pragma unroll
            for (int w = 0; w < GRU_WARPS; ++w) {
                float x[V], y[V];
                Lanes<float, V>::load(&s_a[w][lane * V], x);
                Lanes<float, V>::load(&s_b[w][lane * V], y);
#pragma unroll
                for (int i = 0; i < V; ++i) { Y[i] = fmaf(x[i], Y[i], y[i]); X[i] *= x[i]; }
            }
            Lanes<float, V>::store(p.seg_a + ((int64_t)r * p.nseg + s) * p.width + c0, X);
            Lanes<float, V>::store(p.seg_b + ((int64_t)r * (p.nseg + 1) + s + 1) * p.width + c0, Y);
        }
        return;
    }
    if (!on) return;
    auto apply = [&](const float* pa, const float* pb) {
        float x[V], y[V];
        Lanes<float, V>::load(pa, x);
        Lanes<float, V>::load(pb, y);
#pragma unroll
        for (int i = 0; i < V; ++i) S[i] = fmaf(x[i], S[i], y[i]);
    };
    if (s > 0)
        for (int w = 0; w < GRU_WARPS; ++w) apply(&p_a[w][lane * V], &p_b[w][lane * V]);
    for (int w = 0; w < warp; ++w) apply(&s_a[w][lane * V], &s_b[w][lane * V]);
#pragma unroll
    for (int k = 0; k < GRU_WARP_TOKENS; ++k) {
        if (k < n) {
            float o[V];
#pragma unroll
            for (int i = 0; i < V; ++i) {
                S[i] = fmaf(a[k][i], S[i], b[k][i]);
                o[i] = S[i] * (g[k][i] * gru_sigmoid<T>(g[k][i]));
            }
            Lanes<T, V>::store(p.out + (t0 + k) * p.width + c0, o);
        }
    }
    // the warp that took the row's last token leaves the state (with one segment: every warp has read it before the barrier)
    if (n > 0 && t0 + n == end) Lanes<float, V>::store(st, S);
}

template <typename T, int V>
static int launch_gru(const GruParams<T>& p, int rows, int pass, cudaStream_t stream) {
    if (pass == 0) {
        const int lanes = (p.width + V - 1) / V;
        const int threads = lanes >= 128 ? 128 : (lanes + 31) / 32 * 32;
        return acorn_launch(min_gru_rows_kernel<T, V>, dim3((lanes + threads - 1) / threads, rows), dim3(threads), 0, stream, p);
    }
    constexpr int VS = V > 2 ? 2 : V;                   // a thread's tokens, not its channels, fill its registers
    const int bx = (p.width + 32 * VS - 1) / (32 * VS);
    if (pass == 1)
        return acorn_launch(min_gru_segment_kernel<T, VS, false>, dim3(bx, rows * (p.nseg - 1)), dim3(32 * GRU_WARPS), 0, stream, p);
    return acorn_launch(min_gru_segment_kernel<T, VS, true>, dim3(bx, rows * p.nseg), dim3(32 * GRU_WARPS), 0, stream, p);
}

extern "C" int acorn_min_gru_segment_tokens() { return GRU_SEG; }

// pass 0: a thread walks a row's tokens; passes 1 and 2: rows in nseg segments of GRU_SEG tokens (pass 2 alone with nseg = 1;
// seg_a, seg_b as above otherwise)
extern "C" int acorn_min_gru(const void* proj, int64_t ld, const float* bias, float* state, int64_t slot_stride,
                             int64_t state_off, const int* row_start, const int* row_slot, void* out, int rows, int width,
                             int pass, int nseg, float* seg_a, float* seg_b, int dtype, cudaStream_t stream) {
    if (rows <= 0 || width <= 0) return 0;
    if (pass < 0 || pass > 2 || (pass == 1 && nseg < 2) || (pass == 2 && nseg < 1) || (pass > 0 && nseg > 1 && (!seg_a || !seg_b)) ||
        (int64_t)rows * (pass ? nseg : 1) > 65535)
        return ACORN_ERR_UNSUPPORTED;
    const uintptr_t all = (uintptr_t)proj | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)out | (uintptr_t)seg_a | (uintptr_t)seg_b;
    const bool vec = width % 4 == 0 && ld % 4 == 0 && slot_stride % 4 == 0 && state_off % 4 == 0 && (all & 15) == 0;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        GruParams<T> p;
        p.proj = (const T*)proj; p.ld = ld; p.bias = bias; p.state = state; p.slot_stride = slot_stride;
        p.state_off = state_off; p.row_start = row_start; p.row_slot = row_slot; p.out = (T*)out; p.width = width;
        p.seg_a = seg_a; p.seg_b = seg_b; p.nseg = nseg;
        return vec ? launch_gru<T, 4>(p, rows, pass, stream) : launch_gru<T, 1>(p, rows, pass, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
