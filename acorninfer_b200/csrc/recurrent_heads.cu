// Recurrent mixers with a matrix state per head: what stands before and after the recurrence (delta_rule.cu), and all of it
// in one kernel for rows of a single token.
//
//   delta_heads_prep   gated delta rule with one decay per head, per token: the short causal convolution over time of the
//                      q, k, v channels with silu (inputs before the step's first token from the request's state, whose
//                      rows of a single token it shifts), unit norms x / sqrt(sum x^2 + 1e-6) of q and k (q also times
//                      dim^-1/2), beta = sigmoid(.), log g = -exp(A_log) softplus(. + dt_bias) and g; float32 out
//   linear_heads_prep  gated linear attention, per token: q times dim^-1/2, k, v as they are, and the decay per key channel
//                      sigmoid(z + bias)^(1 / tau); float32 out
//   recurrent_step     rows of one token: a block a (row, head) reads the head's state once, decays it, corrects and writes
//                      (delta rule) or just writes, reads out, norms the result over the head's value channels, multiplies by
//                      a weight and silu of a gate, and stores the state back
#include "common.cuh"

#define RH_MAX_TAPS 16

// pointers that are read four elements at a time: 16-byte aligned float32, 8-byte aligned rows of the activation dtype
static bool rh_aligned(uintptr_t f32_ptrs, uintptr_t rows, int dtype) {
    return (f32_ptrs & 15) == 0 && (rows & (dtype == ACORN_DTYPE_BF16 ? 7 : 15)) == 0;
}

__device__ __forceinline__ float rh_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
// silu where its result goes on in 16 bits' precision anyway (inputs rounded to bfloat16): fast exponential and quotient, relative
// error about 2^-21
template <typename T> __device__ __forceinline__ float rh_silu(float z) { return z * rh_sigmoid(z); }
template <> __device__ __forceinline__ float rh_silu<bf16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ float rh_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
__device__ __forceinline__ float rh_decay(float z, float inv_tau) { return expf(-rh_softplus(-z) * inv_tau); }

template <typename T> struct DeltaHeadsParams {
    const T* in;               // [tokens, ld]: q (KH dim), k (KH dim), v (H vdim) channels; beta's and the decay's columns
    int64_t ld;
    int beta0, decay0;
    const float* conv_w;       // [C, taps] or null: no convolution
    float* state;
    int64_t slot_stride, conv_off;
    const float* A_log;
    const float* dt_bias;
    const int* token_row;
    const int* row_start;
    const int* row_slot;
    float* qn;
    float* kn;
    float* vv;
    float* beta;
    float* g;
    float* log_g;
    int tokens, H, KH, dim, vdim, taps, update_single;
};

// Four channels a lane, 2^lph_log2 lanes a head; a lane takes TPT consecutive tokens, whose inputs and those before them are
// fetched at once.
template <typename T, int TAPS, int TPT>
__global__ void __launch_bounds__(256) delta_heads_prep_vec_kernel(const DeltaHeadsParams<T> p, int lph_log2) {
    constexpr int PAST = TAPS > 1 ? TAPS - 1 : 0;
    const int heads = 2 * p.KH + p.H;
    const int64_t gid = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    const int64_t item = gid >> lph_log2;
    const int l = (int)(gid & ((1 << lph_log2) - 1));
    const int64_t chunks = ((int64_t)p.tokens + TPT - 1) / TPT;
    const bool in_range = item < chunks * heads;
    const int64_t it = in_range ? item : 0;
    const int t0 = (int)(it / heads) * TPT;
    const int h = (int)(it % heads), vh = h - 2 * p.KH;
    const bool is_v = h >= 2 * p.KH;
    const bool lane_on = in_range && 4 * l < (is_v ? p.vdim : p.dim);
    const int C = 2 * p.KH * p.dim + p.H * p.vdim;
    const int chan = lane_on ? (is_v ? 2 * p.KH * p.dim + vh * p.vdim : h * p.dim) + 4 * l : 0;      // idle lanes read channel 0
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float w[TAPS > 0 ? 4 * TAPS : 1];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        const float4 v = *reinterpret_cast<const float4*>(p.conv_w + (int64_t)chan * TAPS + 4 * j);
        w[4 * j] = v.x; w[4 * j + 1] = v.y; w[4 * j + 2] = v.z; w[4 * j + 3] = v.w;
    }
    const bool scalars = is_v && l == 0 && in_range;    // this lane also makes its head's write strength and decay
    float A = 0.f, bias = 0.f;
    if (scalars) {
        A = expf(p.A_log[vh]);
        bias = p.dt_bias[vh];
    }
    pdl_wait();
    pdl_trigger();
    float4 in[TPT + PAST];                              // inputs of tokens t0 - PAST .. t0 + TPT - 1
#pragma unroll
    for (int q = 0; q < TPT + PAST; ++q) {
        const int t = min(max(t0 + q - PAST, 0), p.tokens - 1);
        in[q] = Vec4<T>::load(p.in + (int64_t)t * p.ld + chan);
    }
#pragma unroll
    for (int q = 0; q < TPT; ++q) {
        const int64_t t = t0 + q;
        const bool active = lane_on && t < p.tokens;
        float4 x = in[q + PAST];
        if constexpr (TAPS > 0) {
            x = zero;
            if constexpr (PAST > 0) {
                const int r = p.token_row[min((int)t, p.tokens - 1)];
                const int first = p.row_start[r], i0 = min((int)t, p.tokens - 1) - first;
                float* cstate = i0 < PAST ? p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.conv_off + chan : nullptr;
                float4 before[PAST];
#pragma unroll
                for (int j = 0; j < PAST; ++j) {        // index within the row i0 - PAST + j; negative: before the step
                    float4 u = in[q + j];
                    if (i0 - PAST + j < 0) u = *reinterpret_cast<const float4*>(cstate + (int64_t)(i0 + j) * C);
                    before[j] = u;
                    x.x = fmaf(w[j], u.x, x.x);
                    x.y = fmaf(w[TAPS + j], u.y, x.y);
                    x.z = fmaf(w[2 * TAPS + j], u.z, x.z);
                    x.w = fmaf(w[3 * TAPS + j], u.w, x.w);
                }
                if (active && p.update_single && i0 == 0 && p.row_start[r + 1] - first == 1) {
                    // the row's only token: a lane alone reads and writes its channels
#pragma unroll
                    for (int j = 1; j < PAST; ++j) *reinterpret_cast<float4*>(cstate + (int64_t)(j - 1) * C) = before[j];
                    *reinterpret_cast<float4*>(cstate + (int64_t)(PAST - 1) * C) = in[q + PAST];
                }
            }
            x.x = fmaf(w[TAPS - 1], in[q + PAST].x, x.x);
            x.y = fmaf(w[2 * TAPS - 1], in[q + PAST].y, x.y);
            x.z = fmaf(w[3 * TAPS - 1], in[q + PAST].z, x.z);
            x.w = fmaf(w[4 * TAPS - 1], in[q + PAST].w, x.w);
        }
        x = make_float4(rh_silu<T>(x.x), rh_silu<T>(x.y), rh_silu<T>(x.z), rh_silu<T>(x.w));
        // every lane of the warp takes part in the sums, whatever its head is
        float ss = lane_on ? x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w : 0.f;
        for (int o = (1 << lph_log2) >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (!active) continue;
        float* dst;
        if (is_v) {
            dst = p.vv + (t * p.H + vh) * p.vdim;
            if (scalars) {
                p.beta[t * p.H + vh] = rh_sigmoid(to_float(p.in[t * p.ld + p.beta0 + vh]));
                const float lg = -A * rh_softplus(to_float(p.in[t * p.ld + p.decay0 + vh]) + bias);
                p.g[t * p.H + vh] = expf(lg);
                p.log_g[t * p.H + vh] = lg;
            }
        } else {
            const bool is_q = h < p.KH;
            const float f = rsqrtf(ss + 1e-6f) * (is_q ? rsqrtf((float)p.dim) : 1.f);
            x = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
            dst = is_q ? p.qn + (t * p.KH + h) * p.dim : p.kn + (t * p.KH + h - p.KH) * p.dim;
        }
        *reinterpret_cast<float4*>(dst + 4 * l) = x;
    }
}

// Any sizes: a warp a (token, head), a head's channels in passes of 32.
template <typename T>
__global__ void delta_heads_prep_kernel(const DeltaHeadsParams<T> p) {
    pdl_wait();
    pdl_trigger();
    const int heads = 2 * p.KH + p.H, lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (int64_t)p.tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item % heads);
    const bool is_v = h >= 2 * p.KH;
    const int vh = h - 2 * p.KH, n = is_v ? p.vdim : p.dim;
    const int C = 2 * p.KH * p.dim + p.H * p.vdim;
    const int chan = is_v ? 2 * p.KH * p.dim + vh * p.vdim : h * p.dim;
    const int r = p.token_row[t], i0 = t - p.row_start[r];
    float* cstate = p.conv_w && p.taps > 1 ? p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.conv_off + chan : nullptr;
    const bool shift = cstate && p.update_single && p.row_start[r + 1] - p.row_start[r] == 1;
    const T* src = p.in + (int64_t)t * p.ld + chan;
    float* dst = is_v ? p.vv + ((int64_t)t * p.H + vh) * p.vdim
                      : (h < p.KH ? p.qn + ((int64_t)t * p.KH + h) * p.dim : p.kn + ((int64_t)t * p.KH + h - p.KH) * p.dim);
    float ss = 0.f;
    for (int i = lane; i < n; i += 32) {
        const float own = to_float(src[i]);
        float x = own;
        if (p.conv_w) {
            const float* w = p.conv_w + (int64_t)(chan + i) * p.taps;
            x = 0.f;
            for (int j = 0; j < p.taps - 1; ++j) {
                const int idx = i0 - (p.taps - 1) + j;
                const float in = idx >= 0 ? to_float(src[(int64_t)(idx - i0) * p.ld + i]) : cstate[(int64_t)(p.taps - 1 + idx) * C + i];
                x = fmaf(w[j], in, x);
                if (shift && j > 0) cstate[(int64_t)(j - 1) * C + i] = in;
            }
            if (shift) cstate[(int64_t)(p.taps - 2) * C + i] = own;
            x = fmaf(w[p.taps - 1], own, x);
        }
        x *= rh_sigmoid(x);
        dst[i] = x;
        ss += x * x;
    }
    if (is_v) {
        if (lane == 0) {
            p.beta[(int64_t)t * p.H + vh] = rh_sigmoid(to_float(p.in[(int64_t)t * p.ld + p.beta0 + vh]));
            const float lg = -expf(p.A_log[vh]) * rh_softplus(to_float(p.in[(int64_t)t * p.ld + p.decay0 + vh]) + p.dt_bias[vh]);
            p.g[(int64_t)t * p.H + vh] = expf(lg);
            p.log_g[(int64_t)t * p.H + vh] = lg;
        }
        return;
    }
    const float f = rsqrtf(warp_sum(ss) + 1e-6f) * (h < p.KH ? rsqrtf((float)p.dim) : 1.f);
    for (int i = lane; i < n; i += 32) dst[i] *= f;      // (a lane's own entries)
}

template <typename T, int TAPS> static int launch_delta_heads_vec(const DeltaHeadsParams<T>& p, cudaStream_t stream) {
    const int widest = p.dim > p.vdim ? p.dim : p.vdim;
    int lph_log2 = 0;
    while ((4 << lph_log2) < widest) ++lph_log2;
    const int tpt = p.tokens > 256 ? 4 : 1;
    const int64_t threads = (((int64_t)p.tokens + tpt - 1) / tpt * (2 * p.KH + p.H)) << lph_log2;
    const int block = threads >= 256 ? 256 : 128;
    const dim3 grid((unsigned)((threads + block - 1) / block));
    if (tpt == 1) return acorn_launch(delta_heads_prep_vec_kernel<T, TAPS, 1>, grid, dim3(block), 0, stream, p, lph_log2);
    return acorn_launch(delta_heads_prep_vec_kernel<T, TAPS, 4>, grid, dim3(block), 0, stream, p, lph_log2);
}

template <typename T> static int launch_delta_heads(const DeltaHeadsParams<T>& p, cudaStream_t stream) {
    const int vec_taps = p.conv_w ? p.taps : 0;
    const uintptr_t all = (uintptr_t)p.conv_w | (uintptr_t)p.state | (uintptr_t)p.qn | (uintptr_t)p.kn | (uintptr_t)p.vv;
    if (p.dim % 4 == 0 && p.vdim % 4 == 0 && p.dim <= 128 && p.vdim <= 128 && vec_taps <= 4 && p.ld % 4 == 0 &&
        p.slot_stride % 4 == 0 && p.conv_off % 4 == 0 &&
        rh_aligned(all, (uintptr_t)p.in, sizeof(T) == 2 ? ACORN_DTYPE_BF16 : ACORN_DTYPE_F32)) {
        switch (vec_taps) {
            case 0: return launch_delta_heads_vec<T, 0>(p, stream);
            case 1: return launch_delta_heads_vec<T, 1>(p, stream);
            case 2: return launch_delta_heads_vec<T, 2>(p, stream);
            case 3: return launch_delta_heads_vec<T, 3>(p, stream);
            default: return launch_delta_heads_vec<T, 4>(p, stream);
        }
    }
    const int64_t items = (int64_t)p.tokens * (2 * p.KH + p.H);
    return acorn_launch(delta_heads_prep_kernel<T>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream, p);
}

extern "C" int acorn_delta_heads_prep(const void* in, int64_t ld, int beta0, int decay0, const float* conv_w, int taps, float* state,
                                      int64_t slot_stride, int64_t conv_off, const float* A_log, const float* dt_bias,
                                      const int* token_row, const int* row_start, const int* row_slot, int update_single,
                                      float* qn, float* kn, float* vv, float* beta, float* g, float* log_g, int tokens, int H, int KH, int dim,
                                      int vdim, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (KH < 1 || H < 1 || H % KH || dim < 1 || vdim < 1 || (conv_w && (taps < 1 || taps > RH_MAX_TAPS)) ||
        (int64_t)tokens * (2 * KH + H) > 0x7fffffff)
        return ACORN_ERR_UNSUPPORTED;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        DeltaHeadsParams<T> p;
        p.in = (const T*)in; p.ld = ld; p.beta0 = beta0; p.decay0 = decay0; p.conv_w = conv_w; p.taps = taps; p.state = state;
        p.slot_stride = slot_stride; p.conv_off = conv_off; p.A_log = A_log; p.dt_bias = dt_bias; p.token_row = token_row;
        p.row_start = row_start; p.row_slot = row_slot; p.update_single = update_single; p.qn = qn; p.kn = kn; p.vv = vv;
        p.beta = beta; p.g = g; p.log_g = log_g; p.tokens = tokens; p.H = H; p.KH = KH; p.dim = dim; p.vdim = vdim;
        return launch_delta_heads<T>(p, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------- gated linear attention

// V: entries a thread (4: 8- or 16-byte accesses; 1 otherwise); a thread's entries are of q, k and the decay, or of v
template <typename T, int V>
__global__ void linear_heads_prep_kernel(const T* __restrict__ in, int64_t ld, const float* __restrict__ z, int64_t ldz,
                                         const float* __restrict__ bias, float inv_tau, float q_scale, float* __restrict__ qn,
                                         float* __restrict__ kn, float* __restrict__ vv, float* __restrict__ alpha, int Hd,
                                         int Hv, int64_t total) {
    pdl_wait();
    pdl_trigger();
    const int per = (Hd + Hv) / V;                      // a token's items: Hd / V of q, k, decay, then Hv / V of v
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / per;
        const int c = (int)(i - t * per) * V;
        const T* row = in + t * ld;
        if constexpr (V == 4) {
            if (c >= Hd) {
                *reinterpret_cast<float4*>(vv + t * Hv + c - Hd) = Vec4<T>::load(row + Hd + c);
                continue;
            }
            const float4 q = Vec4<T>::load(row + c), zz = *reinterpret_cast<const float4*>(z + t * ldz + c),
                         b = *reinterpret_cast<const float4*>(bias + c);
            *reinterpret_cast<float4*>(kn + t * Hd + c) = Vec4<T>::load(row + Hd + c);
            *reinterpret_cast<float4*>(qn + t * Hd + c) = make_float4(q.x * q_scale, q.y * q_scale, q.z * q_scale, q.w * q_scale);
            *reinterpret_cast<float4*>(alpha + t * Hd + c) =
                make_float4(rh_decay(zz.x + b.x, inv_tau), rh_decay(zz.y + b.y, inv_tau), rh_decay(zz.z + b.z, inv_tau),
                            rh_decay(zz.w + b.w, inv_tau));
        } else {
            if (c >= Hd) {
                vv[t * Hv + c - Hd] = to_float(row[Hd + c]);
                continue;
            }
            qn[t * Hd + c] = to_float(row[c]) * q_scale;
            kn[t * Hd + c] = to_float(row[Hd + c]);
            alpha[t * Hd + c] = rh_decay(z[t * ldz + c] + bias[c], inv_tau);
        }
    }
}

// in: a token's [q (H dim) | k (H dim) | v (H vdim)]; z [tokens, ldz] float32 the decays' pre-activations
extern "C" int acorn_linear_heads_prep(const void* in, int64_t ld, const float* z, int64_t ldz, const float* bias, float inv_tau,
                                       float* qn, float* kn, float* vv, float* alpha, int tokens, int H, int dim, int vdim,
                                       int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (H < 1 || dim < 1 || vdim < 1) return ACORN_ERR_UNSUPPORTED;
    const int Hd = H * dim, Hv = H * vdim;
    const float q_scale = (float)(1.0 / sqrt((double)dim));
    const uintptr_t all = (uintptr_t)z | (uintptr_t)bias | (uintptr_t)qn | (uintptr_t)kn | (uintptr_t)vv | (uintptr_t)alpha;
    const bool vec = Hd % 4 == 0 && Hv % 4 == 0 && ld % 4 == 0 && ldz % 4 == 0 && rh_aligned(all, (uintptr_t)in, dtype);
    const int64_t total = (int64_t)tokens * (Hd + Hv) / (vec ? 4 : 1);
    int64_t blocks = (total + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    if (vec)
        ACORN_DISPATCH_DTYPE(dtype, T, return acorn_launch(linear_heads_prep_kernel<T, 4>, dim3((unsigned)blocks), dim3(256), 0, stream,
                                                           (const T*)in, ld, z, ldz, bias, inv_tau, q_scale, qn, kn, vv, alpha, Hd, Hv, total));
    ACORN_DISPATCH_DTYPE(dtype, T, return acorn_launch(linear_heads_prep_kernel<T, 1>, dim3((unsigned)blocks), dim3(256), 0, stream,
                                                       (const T*)in, ld, z, ldz, bias, inv_tau, q_scale, qn, kn, vv, alpha, Hd, Hv, total));
    return ACORN_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------- rows of one token

#define RS_WARPS 8

template <typename T> struct StepParams {
    // delta rule: q, k [rows, KH, dim], v [rows, H, vdim], beta, decay [rows, H], float32
    const float* q;
    const float* k;
    const float* v;
    const float* beta;
    const float* decay;
    // linear attention: the projected row [q | k | v] and the decays' pre-activations
    const T* in;
    int64_t ld;
    const float* z;
    int64_t ldz;
    const float* bias;
    float inv_tau, q_scale;
    const T* gate;             // [rows, ldg]: head h's gate at column h vdim
    int64_t ldg;
    const float* norm_w;       // [vdim]
    float eps, out_scale;
    float* state;
    int64_t slot_stride;
    const int* row_slot;
    T* out;
    int64_t ldo;
    int H, KH, dim, vdim;
};

// A block a (row, head).  A warp takes every RS_WARPS-th row of the state (a key channel), a lane VV vectors of four value
// channels of it; all of the head's state is in registers (DR rows a warp) between its one read and its one write.
//     a = S'^T k, b = S'^T q with S' = g S;   u = beta (v - a) or v;   o = b + (k . q) u;   S = S' + k u^T
template <typename T, bool RULE, int DR, int VV>
__global__ void __launch_bounds__(RS_WARPS * 32) recurrent_step_kernel(const StepParams<T> p) {
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                                     // [dim] q, k, decays
    float* sk = sq + p.dim;
    float* sg = sk + p.dim;
    float4* pa = reinterpret_cast<float4*>(sm + (3 * p.dim + 3) / 4 * 4);       // [RS_WARPS][VV * 32]
    float4* pb = pa + RS_WARPS * VV * 32;
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* S_g = p.state + (int64_t)p.row_slot[r] * p.slot_stride + (int64_t)h * p.dim * p.vdim;
    float4 S[DR][VV];
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int d = warp + RS_WARPS * i;
#pragma unroll
        for (int c = 0; c < VV; ++c) {
            const int col = 4 * (lane + 32 * c);
            S[i][c] = d < p.dim && col < p.vdim ? *reinterpret_cast<const float4*>(S_g + (int64_t)d * p.vdim + col)
                                                : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    float4 v[VV], z[VV], w[VV];
#pragma unroll
    for (int c = 0; c < VV; ++c) {
        const int col = 4 * (lane + 32 * c);
        v[c] = z[c] = w[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (col < p.vdim) {
            v[c] = RULE ? *reinterpret_cast<const float4*>(p.v + ((int64_t)r * p.H + h) * p.vdim + col)
                        : Vec4<T>::load(p.in + (int64_t)r * p.ld + 2 * p.H * p.dim + h * p.vdim + col);
            z[c] = Vec4<T>::load(p.gate + (int64_t)r * p.ldg + h * p.vdim + col);
            w[c] = *reinterpret_cast<const float4*>(p.norm_w + col);
        }
    }
    float beta = 1.f;
    if constexpr (RULE) {
        const float g = p.decay[(int64_t)r * p.H + h];
        beta = p.beta[(int64_t)r * p.H + h];
        const int kh = h / (p.H / p.KH);
        for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
            sq[d] = p.q[((int64_t)r * p.KH + kh) * p.dim + d];
            sk[d] = p.k[((int64_t)r * p.KH + kh) * p.dim + d];
            sg[d] = g;
        }
    } else {
        for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
            const int c = h * p.dim + d;
            sq[d] = to_float(p.in[(int64_t)r * p.ld + c]) * p.q_scale;
            sk[d] = to_float(p.in[(int64_t)r * p.ld + p.H * p.dim + c]);
            sg[d] = rh_decay(p.z[(int64_t)r * p.ldz + c] + p.bias[c], p.inv_tau);
        }
    }
    __syncthreads();
    float kq = 0.f;                                     // every warp sums all of it
    for (int d = lane; d < p.dim; d += 32) kq = fmaf(sq[d], sk[d], kq);
    kq = warp_sum(kq);
    float4 a[VV], b[VV];
#pragma unroll
    for (int c = 0; c < VV; ++c) a[c] = b[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int d = warp + RS_WARPS * i;
        const float g = d < p.dim ? sg[d] : 0.f, k = d < p.dim ? sk[d] : 0.f, q = d < p.dim ? sq[d] : 0.f;
#pragma unroll
        for (int c = 0; c < VV; ++c) {
            float4& s = S[i][c];
            s.x *= g; s.y *= g; s.z *= g; s.w *= g;
            if (RULE) {
                a[c].x = fmaf(k, s.x, a[c].x); a[c].y = fmaf(k, s.y, a[c].y);
                a[c].z = fmaf(k, s.z, a[c].z); a[c].w = fmaf(k, s.w, a[c].w);
            }
            b[c].x = fmaf(q, s.x, b[c].x); b[c].y = fmaf(q, s.y, b[c].y);
            b[c].z = fmaf(q, s.z, b[c].z); b[c].w = fmaf(q, s.w, b[c].w);
        }
    }
#pragma unroll
    for (int c = 0; c < VV; ++c) {
        if (RULE) pa[(warp * VV + c) * 32 + lane] = a[c];
        pb[(warp * VV + c) * 32 + lane] = b[c];
    }
    __syncthreads();
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < VV; ++c) {                      // every warp: the sums over all key channels, u and o of the lane's columns
        a[c] = b[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int q = 0; q < RS_WARPS; ++q) {
            if (RULE) {
                const float4 e = pa[(q * VV + c) * 32 + lane];
                a[c].x += e.x; a[c].y += e.y; a[c].z += e.z; a[c].w += e.w;
            }
            const float4 f = pb[(q * VV + c) * 32 + lane];
            b[c].x += f.x; b[c].y += f.y; b[c].z += f.z; b[c].w += f.w;
        }
        // a becomes u, b the read-out
        a[c] = RULE ? make_float4(beta * (v[c].x - a[c].x), beta * (v[c].y - a[c].y), beta * (v[c].z - a[c].z), beta * (v[c].w - a[c].w)) : v[c];
        b[c].x = fmaf(kq, a[c].x, b[c].x); b[c].y = fmaf(kq, a[c].y, b[c].y);
        b[c].z = fmaf(kq, a[c].z, b[c].z); b[c].w = fmaf(kq, a[c].w, b[c].w);
        ss += b[c].x * b[c].x + b[c].y * b[c].y + b[c].z * b[c].z + b[c].w * b[c].w;
    }
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int d = warp + RS_WARPS * i;
        if (d >= p.dim) break;
        const float k = sk[d];
#pragma unroll
        for (int c = 0; c < VV; ++c) {
            const int col = 4 * (lane + 32 * c);
            if (col < p.vdim)
                *reinterpret_cast<float4*>(S_g + (int64_t)d * p.vdim + col) =
                    make_float4(fmaf(k, a[c].x, S[i][c].x), fmaf(k, a[c].y, S[i][c].y), fmaf(k, a[c].z, S[i][c].z), fmaf(k, a[c].w, S[i][c].w));
        }
    }
    if (warp != 0) return;
    const float inv = rsqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
#pragma unroll
    for (int c = 0; c < VV; ++c) {
        const int col = 4 * (lane + 32 * c);
        if (col >= p.vdim) break;
        auto one = [&](float o, float wt, float zz) { return o * inv * wt * (zz * rh_sigmoid(zz)) * p.out_scale; };
        Vec4<T>::store(p.out + (int64_t)r * p.ldo + h * p.vdim + col,
                       make_float4(one(b[c].x, w[c].x, z[c].x), one(b[c].y, w[c].y, z[c].y), one(b[c].z, w[c].z, z[c].z),
                                   one(b[c].w, w[c].w, z[c].w)));
    }
}

extern "C" int acorn_recurrent_step_supported(int dim, int vdim) {
    return dim >= 1 && dim <= 256 && vdim >= 4 && vdim % 4 == 0 && (vdim <= 128 || (vdim <= 256 && dim <= 128));
}

template <typename T, bool RULE> static int launch_step(const StepParams<T>& p, int rows, cudaStream_t stream) {
    const int vv = p.vdim <= 128 ? 1 : 2;
    const size_t smem = ((size_t)(3 * p.dim + 3) / 4 * 4 + (size_t)2 * RS_WARPS * vv * 32 * 4) * sizeof(float);
    const dim3 grid(rows, p.H), block(RS_WARPS * 32);
#define STEP(DR, VV) return acorn_launch(recurrent_step_kernel<T, RULE, DR, VV>, grid, block, smem, stream, p)
    if (vv == 1) {
        if (p.dim <= 32) STEP(4, 1);
        if (p.dim <= 64) STEP(8, 1);
        if (p.dim <= 128) STEP(16, 1);
        STEP(32, 1);
    }
    if (p.dim <= 64) STEP(8, 2);
    STEP(16, 2);
#undef STEP
}

extern "C" int acorn_recurrent_step(int rule, const float* q, const float* k, const float* v, const float* beta, const float* decay,
                                    const void* in, int64_t ld, const float* z, int64_t ldz, const float* bias, float inv_tau,
                                    const void* gate, int64_t ldg, const float* norm_w, float eps, float out_scale, float* state,
                                    int64_t slot_stride, const int* row_slot, void* out, int64_t ldo, int rows, int H, int KH,
                                    int dim, int vdim, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (!acorn_recurrent_step_supported(dim, vdim) || H < 1 || H > 65535 || KH < 1 || H % KH || slot_stride % 4 ||
        !rh_aligned((uintptr_t)v | (uintptr_t)norm_w | (uintptr_t)state, (uintptr_t)in | (uintptr_t)gate | (uintptr_t)out, dtype) ||
        ldg % 4 || ldo % 4 || (!rule && (ld % 4 || (H * dim) % 2)))
        return ACORN_ERR_UNSUPPORTED;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        StepParams<T> p;
        p.q = q; p.k = k; p.v = v; p.beta = beta; p.decay = decay; p.in = (const T*)in; p.ld = ld; p.z = z; p.ldz = ldz;
        p.bias = bias; p.inv_tau = inv_tau; p.q_scale = (float)(1.0 / sqrt((double)dim)); p.gate = (const T*)gate; p.ldg = ldg;
        p.norm_w = norm_w; p.eps = eps; p.out_scale = out_scale; p.state = state; p.slot_stride = slot_stride;
        p.row_slot = row_slot; p.out = (T*)out; p.ldo = ldo; p.H = H; p.KH = KH; p.dim = dim; p.vdim = vdim;
        return rule ? launch_step<T, true>(p, rows, stream) : launch_step<T, false>(p, rows, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
