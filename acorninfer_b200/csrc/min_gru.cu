// A gated recurrence whose gates read the current token only (minGRU), over every row's tokens, channel by channel:
//
//   z = sigmoid(proj_z + b_z),   u = proj_u + b_u,   c = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S <- (1 - z) S + z c                             float32, in the request's state slot between steps
//   out = S * silu(proj_g)
//
// proj holds [z | u | g] of `width` columns each, as projected.  A thread takes V neighbouring channels.  Rows of a few
// tokens: a thread walks its channels (min_gru_rows).  Longer rows take two passes, both over chunks of GRU_CHUNK tokens a warp
// whose loads are all in flight at once.  A token maps S to a S + b, and maps compose.  First (min_gru_maps): a block takes a
// segment of the row, GRU_WARPS chunks at a time; the chunks' maps meet in shared memory, and what is left in memory
// is every chunk's map of the tokens before it in its segment, every segment's own map, and the row's state before the step.
// Second (min_gru_outputs): a warp a chunk composes the maps of the segments before (at most GRU_MAX_SEGMENTS) and of the
// chunks before, and walks its tokens; the last chunk of a row leaves the state.
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
    float* pre_a;             // [rows, nchunks, width] the map of the tokens before a chunk in its segment
    float* pre_b;
    int nchunks, seg_chunks;  // chunks of the longest row; chunks of a segment, a multiple of GRU_WARPS
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
template <typename T> __device__ __forceinline__ void gru_gates(float z_in, float u, float& z, float& c);
template <> __device__ __forceinline__ void gru_gates<float>(float z_in, float u, float& z, float& c) {
    z = gru_sigmoid<float>(z_in);
    c = u >= 0.f ? u + 0.5f : gru_sigmoid<float>(u);
}
// both sigmoids from one reciprocal; below -40 a sigmoid is less than 5e-18
template <> __device__ __forceinline__ void gru_gates<bf16>(float z_in, float u, float& z, float& c) {
    const float e1 = 1.f + __expf(-fmaxf(z_in, -40.f)), e2 = 1.f + __expf(-fmaxf(u, -40.f));
    const float r = __fdividef(1.f, e1 * e2);
    z = r * e2;
    c = u >= 0.f ? u + 0.5f : r * e1;
}

#define GRU_CHUNK 8
#define GRU_WARPS 16
#define GRU_MAX_SEGMENTS 16

// the tokens t0 .. t0 + n - 1 (1 <= n <= GRU_CHUNK): S on, outputs written.  The loads of all GRU_CHUNK are issued without a
// condition between them (beyond n the last token's again), so that they are in flight together.
template <typename T, int V>
__device__ __forceinline__ void gru_walk(const GruParams<T>& p, int c0, int64_t t0, int n, const float (&bz)[V],
                                         const float (&bu)[V], float (&S)[V]) {
    float z[GRU_CHUNK][V], u[GRU_CHUNK][V], g[GRU_CHUNK][V];
#pragma unroll
    for (int k = 0; k < GRU_CHUNK; ++k) {
        const T* row = p.proj + (t0 + min(k, n - 1)) * p.ld + c0;
        Lanes<T, V>::load(row, z[k]);
        Lanes<T, V>::load(row + p.width, u[k]);
        Lanes<T, V>::load(row + 2 * (int64_t)p.width, g[k]);
    }
#pragma unroll
    for (int k = 0; k < GRU_CHUNK; ++k) {
#pragma unroll
        for (int i = 0; i < V; ++i) {
            float zz, cc;
            gru_gates<T>(z[k][i] + bz[i], u[k][i] + bu[i], zz, cc);
            const float next = fmaf(1.f - zz, S[i], zz * cc);
            S[i] = k < n ? next : S[i];
            g[k][i] = S[i] * (g[k][i] * gru_sigmoid<T>(g[k][i]));
        }
        if (k < n) Lanes<T, V>::store(p.out + (t0 + k) * p.width + c0, g[k]);
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
    const int64_t end = p.row_start[r + 1];
    for (int64_t t = p.row_start[r]; t < end; t += GRU_CHUNK)
        gru_walk<T, V>(p, c0, t, (int)min((int64_t)GRU_CHUNK, end - t), bz, bu, S);
    Lanes<float, V>::store(st, S);
}

// blockIdx.y = row * nseg + segment
template <typename T, int V>
__global__ void __launch_bounds__(32 * GRU_WARPS, 2) min_gru_maps_kernel(const GruParams<T> p) {
    __shared__ __align__(16) float s_a[2][GRU_WARPS][32 * V], s_b[2][GRU_WARPS][32 * V];    // the chunks' maps, of two rounds
    pdl_wait();
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = blockIdx.y / p.nseg, s = blockIdx.y % p.nseg;
    const int c0 = (blockIdx.x * 32 + lane) * V;
    const bool on = c0 < p.width;
    const int c_load = on ? c0 : p.width - V;
    const int64_t first = p.row_start[r], end = p.row_start[r + 1];
    const int64_t seg0 = first + (int64_t)s * p.seg_chunks * GRU_CHUNK;
    if (s == 0 && warp == 0 && on) {
        float S[V];
        Lanes<float, V>::load(p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0, S);
        Lanes<float, V>::store(p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0, S);
    }
    float bz[V], bu[V], X[V], Y[V];                     // X, Y: the map of the segment's tokens before this round
#pragma unroll
    for (int i = 0; i < V; ++i) { X[i] = 1.f; Y[i] = 0.f; }
    Lanes<float, V>::load(p.bias + c_load, bz);
    Lanes<float, V>::load(p.bias + p.width + c_load, bu);
    for (int round = 0; round * GRU_WARPS < p.seg_chunks; ++round) {
        const int64_t r0 = seg0 + (int64_t)round * GRU_WARPS * GRU_CHUNK;
        if (r0 >= end) break;                           // (the same for the whole block)
        const int64_t t0 = r0 + warp * GRU_CHUNK;
        const int n = on ? (int)max((int64_t)0, min((int64_t)GRU_CHUNK, end - t0)) : 0;
        float z[GRU_CHUNK][V], u[GRU_CHUNK][V], A[V], B[V];
        // without a condition between them, so that they are in flight together: beyond the row its last token, beyond the
        // width the last channels, neither of which counts
#pragma unroll
        for (int k = 0; k < GRU_CHUNK; ++k) {
            const T* row = p.proj + min(t0 + k, end - 1) * p.ld + c_load;
            Lanes<T, V>::load(row, z[k]);
            Lanes<T, V>::load(row + p.width, u[k]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) { A[i] = 1.f; B[i] = 0.f; }
#pragma unroll
        for (int k = 0; k < GRU_CHUNK; ++k) {
#pragma unroll
            for (int i = 0; i < V; ++i) {
                float zz, cc;
                gru_gates<T>(z[k][i] + bz[i], u[k][i] + bu[i], zz, cc);
                zz = k < n ? zz : 0.f;                  // a map that changes nothing
                A[i] *= 1.f - zz;
                B[i] = fmaf(1.f - zz, B[i], zz * cc);
            }
        }
        Lanes<float, V>::store(&s_a[round & 1][warp][lane * V], A);
        Lanes<float, V>::store(&s_b[round & 1][warp][lane * V], B);
        __syncthreads();                                // (the buffer of the round before may still be read)
#pragma unroll
        for (int w = 0; w < GRU_WARPS; ++w) {
            if (w == warp && n > 0) {
                const int64_t at = ((int64_t)r * p.nchunks + (t0 - first) / GRU_CHUNK) * p.width + c0;
                Lanes<float, V>::store(p.pre_a + at, X);
                Lanes<float, V>::store(p.pre_b + at, Y);
            }
            float x[V], y[V];
            Lanes<float, V>::load(&s_a[round & 1][w][lane * V], x);
            Lanes<float, V>::load(&s_b[round & 1][w][lane * V], y);
#pragma unroll
            for (int i = 0; i < V; ++i) { Y[i] = fmaf(x[i], Y[i], y[i]); X[i] *= x[i]; }
        }
    }
    if (warp == 0 && on && seg0 < end) {
        Lanes<float, V>::store(p.seg_a + ((int64_t)r * p.nseg + s) * p.width + c0, X);
        Lanes<float, V>::store(p.seg_b + ((int64_t)r * (p.nseg + 1) + s + 1) * p.width + c0, Y);
    }
}

#define GRU_OUT_WARPS 4

// blockIdx.y = row * blocks of a row + block of GRU_OUT_WARPS chunks
template <typename T, int V>
__global__ void __launch_bounds__(32 * GRU_OUT_WARPS) min_gru_outputs_kernel(const GruParams<T> p) {
    pdl_wait();
    pdl_trigger();
    const int per_row = (p.nchunks + GRU_OUT_WARPS - 1) / GRU_OUT_WARPS;
    const int r = blockIdx.y / per_row, chunk = blockIdx.y % per_row * GRU_OUT_WARPS + (threadIdx.x >> 5);
    const int c0 = (blockIdx.x * 32 + (threadIdx.x & 31)) * V;
    const int64_t first = p.row_start[r], end = p.row_start[r + 1], t0 = first + (int64_t)chunk * GRU_CHUNK;
    if (c0 >= p.width || t0 >= end) return;
    const float* sa = p.seg_a + (int64_t)r * p.nseg * p.width + c0;
    const float* sb = p.seg_b + (int64_t)r * (p.nseg + 1) * p.width + c0;
    const int64_t at = ((int64_t)r * p.nchunks + chunk) * p.width + c0;
    float bz[V], bu[V], S[V], x[V], y[V];
    Lanes<float, V>::load(p.bias + c0, bz);
    Lanes<float, V>::load(p.bias + p.width + c0, bu);
    Lanes<float, V>::load(sb, S);
    const int s = chunk / p.seg_chunks;
#pragma unroll 4
    for (int q = 0; q < s; ++q) {
        Lanes<float, V>::load(sa + (int64_t)q * p.width, x);
        Lanes<float, V>::load(sb + (int64_t)(q + 1) * p.width, y);
#pragma unroll
        for (int i = 0; i < V; ++i) S[i] = fmaf(x[i], S[i], y[i]);
    }
    Lanes<float, V>::load(p.pre_a + at, x);
    Lanes<float, V>::load(p.pre_b + at, y);
#pragma unroll
    for (int i = 0; i < V; ++i) S[i] = fmaf(x[i], S[i], y[i]);
    const int n = (int)min((int64_t)GRU_CHUNK, end - t0);
    gru_walk<T, V>(p, c0, t0, n, bz, bu, S);
    if (t0 + n == end) Lanes<float, V>::store(p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.state_off + c0, S);
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
        return acorn_launch(min_gru_maps_kernel<T, VS>, dim3(bx, rows * p.nseg), dim3(32 * GRU_WARPS), 0, stream, p);
    return acorn_launch(min_gru_outputs_kernel<T, VS>, dim3(bx, rows * ((p.nchunks + GRU_OUT_WARPS - 1) / GRU_OUT_WARPS)),
                        dim3(32 * GRU_OUT_WARPS), 0, stream, p);
}

// pass 0: a thread walks a row's tokens; passes 1 and 2: rows of up to longest_row tokens in chunks (segs: float32 memory of
// acorn_min_gru_scratch floats)
extern "C" int64_t acorn_min_gru_scratch(int rows, int width, int longest_row) {
    const int64_t nchunks = (longest_row + GRU_CHUNK - 1) / GRU_CHUNK;
    return (int64_t)rows * width * (2 * nchunks + 2 * GRU_MAX_SEGMENTS + 1);
}

extern "C" int acorn_min_gru(const void* proj, int64_t ld, const float* bias, float* state, int64_t slot_stride,
                             int64_t state_off, const int* row_start, const int* row_slot, void* out, int rows, int width,
                             int pass, int longest_row, float* scratch, int dtype, cudaStream_t stream) {
    if (rows <= 0 || width <= 0) return 0;
    if (pass < 0 || pass > 2 || (pass > 0 && (longest_row < 1 || !scratch))) return ACORN_ERR_UNSUPPORTED;
    const int nchunks = pass ? (longest_row + GRU_CHUNK - 1) / GRU_CHUNK : 1;
    const int seg_chunks = GRU_WARPS * ((nchunks + GRU_WARPS * GRU_MAX_SEGMENTS - 1) / (GRU_WARPS * GRU_MAX_SEGMENTS));
    const int nseg = (nchunks + seg_chunks - 1) / seg_chunks;
    if ((int64_t)rows * nchunks > 65535 || rows > 65535) return ACORN_ERR_UNSUPPORTED;
    const uintptr_t all = (uintptr_t)proj | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)out | (uintptr_t)scratch;
    const bool vec = width % 4 == 0 && ld % 4 == 0 && slot_stride % 4 == 0 && state_off % 4 == 0 && (all & 15) == 0;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        GruParams<T> p;
        p.proj = (const T*)proj; p.ld = ld; p.bias = bias; p.state = state; p.slot_stride = slot_stride;
        p.state_off = state_off; p.row_start = row_start; p.row_slot = row_slot; p.out = (T*)out; p.width = width;
        p.nchunks = nchunks; p.seg_chunks = seg_chunks; p.nseg = nseg;
        const int64_t line = (int64_t)rows * width;
        p.pre_a = scratch; p.pre_b = scratch + line * nchunks;
        p.seg_a = scratch + 2 * line * nchunks; p.seg_b = p.seg_a + line * nseg;
        return vec ? launch_gru<T, 4>(p, rows, pass, stream) : launch_gru<T, 1>(p, rows, pass, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
