// What lies between the projection and the attention where q and k are normed over the whole projected row (all heads
// together) and not per head.  Per token, from its row [q: nq d | k: nkv d | v: nkv dv], in float32:
//   bias, short causal convolution over time per channel (as in qk_rope_kv.cu: the last taps - 1 inputs of a request are
//   kept in its state slot, [taps - 1, channels] in time order);
//   q <- q * rsqrt(sum(q^2) / q_count + eps) * q_w, k likewise over its own row (q_count, k_count: how many of a row's
//   entries count, where heads are padded with zeros);
//   the first `rot` entries of every q and k head rotated by the step's table of cosines and sines
//   ([tokens, rot]: rot / 2 cosines, then the sines); pairs (2i, 2i + 1), or (i, i + rot / 2) with `pairing` 0;
//   q to q_out, k and v (times v_scale) into the request's pages.
#include "common.cuh"

#define ROWN_MAX_TAPS 16

template <typename T> struct RowNormParams {
    const T* proj;
    int64_t ld;
    T* q_out;
    int64_t ld_q;
    T* k_pages;
    T* v_pages;
    const float* q_w;          // [nq d] or null: no norm
    const float* k_w;          // [nkv d] or null
    const float* conv_w;       // [channels, taps] or null
    const float* bias;         // [channels] or null
    float* state;
    int64_t slot_stride, conv_off;
    const int* row_start;
    const int* row_slot;
    const int* token_row;
    const int* positions;
    const int* block_table;
    const int* page_base;
    int table_stride;
    const float* cos_sin;      // [tokens, rot] or null with rot 0
    int tokens, nq, nkv, d, dv, P, rot, pairing, taps, update_single;
    float q_count, k_count, eps, v_scale;
};

__device__ __forceinline__ void rown_pair_sum(float& a, float& b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    const float2 t = lane < nwarps ? scratch[lane] : make_float2(0.f, 0.f);
    a = warp_sum(t.x);
    b = warp_sum(t.y);
}

// Four channels a lane, VPT such vectors a thread; a block takes TPT consecutive tokens of the step: their rows and those before
// them are fetched at once, the convolved values wait in registers for the rows' norms.
template <typename T, int TAPS, int VPT, int TPT>
__global__ void __launch_bounds__(VPT == 1 ? 768 : 512) qk_row_norm_vec_kernel(const RowNormParams<T> p) {
    __shared__ float sums[2 * TPT][32];
    __shared__ float inv_s[2 * TPT];
    constexpr int PAST = TAPS > 1 ? TAPS - 1 : 0;
    constexpr int WT = TAPS > 0 ? 4 * TAPS : 1;
    const int qv = p.nq * p.d / 4, kv = p.nkv * p.d / 4, nvec = qv + kv + p.nkv * p.dv / 4;
    const int channels = nvec * 4;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int t0 = blockIdx.x * TPT;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 x[VPT][TPT];
    int chan[VPT], kind[VPT];                           // kind 0: q, 1: k, 2: v, 3: no vector
    float sq[TPT], sk[TPT];
#pragma unroll
    for (int q = 0; q < TPT; ++q) sq[q] = sk[q] = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int v = threadIdx.x + k * blockDim.x;
        kind[k] = v >= nvec ? 3 : (v >= qv + kv ? 2 : (v >= qv ? 1 : 0));
        chan[k] = 4 * min(v, nvec - 1);
    }
    int row[TPT], i0[TPT];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        float w[WT];
        const float4 b = p.bias ? *reinterpret_cast<const float4*>(p.bias + chan[k]) : zero;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const float4 u = *reinterpret_cast<const float4*>(p.conv_w + (int64_t)chan[k] * TAPS + 4 * j);
            w[4 * j] = u.x; w[4 * j + 1] = u.y; w[4 * j + 2] = u.z; w[4 * j + 3] = u.w;
        }
        if (k == 0) {
            pdl_wait();
            pdl_trigger();
#pragma unroll
            for (int q = 0; q < TPT; ++q) {
                const int t = min(t0 + q, p.tokens - 1);
                row[q] = p.token_row[t];
                i0[q] = PAST ? t - p.row_start[row[q]] : 0;               // the token's index within its row
            }
        }
        float4 in[TPT + PAST];                          // inputs of tokens t0 - PAST .. t0 + TPT - 1
#pragma unroll
        for (int q = 0; q < TPT + PAST; ++q) {
            const int t = min(max(t0 + q - PAST, 0), p.tokens - 1);
            const float4 u = Vec4<T>::load(p.proj + (int64_t)t * p.ld + chan[k]);
            in[q] = make_float4(u.x + b.x, u.y + b.y, u.z + b.z, u.w + b.w);
        }
#pragma unroll
        for (int q = 0; q < TPT; ++q) {
            float4 y = in[q + PAST];
            if constexpr (TAPS > 0) {
                y = zero;
                float* cstate = nullptr;
                if constexpr (PAST > 0)
                    if (i0[q] < PAST) cstate = p.state + (int64_t)p.row_slot[row[q]] * p.slot_stride + p.conv_off + chan[k];
                float4 before[PAST > 0 ? PAST : 1];
#pragma unroll
                for (int j = 0; j < PAST; ++j) {        // index within the row i0 - PAST + j; negative: before the step
                    float4 u = in[q + j];
                    if (i0[q] - PAST + j < 0) u = *reinterpret_cast<const float4*>(cstate + (int64_t)(i0[q] + j) * channels);
                    before[j] = u;
                    y.x = fmaf(w[j], u.x, y.x);
                    y.y = fmaf(w[TAPS + j], u.y, y.y);
                    y.z = fmaf(w[2 * TAPS + j], u.z, y.z);
                    y.w = fmaf(w[3 * TAPS + j], u.w, y.w);
                }
                y.x = fmaf(w[TAPS - 1], in[q + PAST].x, y.x);
                y.y = fmaf(w[2 * TAPS - 1], in[q + PAST].y, y.y);
                y.z = fmaf(w[3 * TAPS - 1], in[q + PAST].z, y.z);
                y.w = fmaf(w[4 * TAPS - 1], in[q + PAST].w, y.w);
                if constexpr (PAST > 0) {
                    // the row's only token: a lane alone reads and writes its channels
                    if (p.update_single && kind[k] < 3 && i0[q] == 0 && t0 + q < p.tokens && p.row_start[row[q] + 1] - (t0 + q) == 1) {
#pragma unroll
                        for (int j = 1; j < PAST; ++j) *reinterpret_cast<float4*>(cstate + (int64_t)(j - 1) * channels) = before[j];
                        *reinterpret_cast<float4*>(cstate + (int64_t)(PAST - 1) * channels) = in[q + PAST];
                    }
                }
            }
            x[k][q] = y;
            const float ss = y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
            if (kind[k] == 0) sq[q] += ss;
            if (kind[k] == 1) sk[q] += ss;
        }
    }
#pragma unroll
    for (int q = 0; q < TPT; ++q) {
        const float a = warp_sum(sq[q]), b = warp_sum(sk[q]);
        if (lane == 0) {
            sums[2 * q][warp] = a;
            sums[2 * q + 1][warp] = b;
        }
    }
    __syncthreads();
    for (int e = warp; e < 2 * TPT; e += nwarps) {
        const float total = warp_sum(lane < nwarps ? sums[e][lane] : 0.f);
        if (lane == 0) inv_s[e] = rsqrtf(total / (e & 1 ? p.k_count : p.q_count) + p.eps);
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < TPT; ++q) {
        const int t = t0 + q;
        if (t >= p.tokens) break;
        const int pos = p.positions[t];
        const int page = p.block_table[(int64_t)row[q] * p.table_stride + (pos / p.P - p.page_base[row[q]])];
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            if (kind[k] == 3) continue;
            float4 y = x[k][q];
            T* dst;
            if (kind[k] == 2) {
                const int c = chan[k] - (p.nq + p.nkv) * p.d;
                const int h = c / p.dv, i = c - h * p.dv;
                y = make_float4(y.x * p.v_scale, y.y * p.v_scale, y.z * p.v_scale, y.w * p.v_scale);
                dst = p.v_pages + (((int64_t)page * p.nkv + h) * p.P + pos % p.P) * p.dv + i;
            } else {
                const int c = kind[k] == 0 ? chan[k] : chan[k] - p.nq * p.d;
                const int h = c / p.d, i = c - h * p.d;
                const float* nw = kind[k] == 0 ? p.q_w : p.k_w;
                if (nw) {
                    const float4 g = *reinterpret_cast<const float4*>(nw + c);
                    const float inv = inv_s[2 * q + kind[k]];
                    y = make_float4(y.x * inv * g.x, y.y * inv * g.y, y.z * inv * g.z, y.w * inv * g.w);
                }
                if (i < p.rot) {                                          // two whole pairs, or one where the rotated part ends between them
                    const float* cs = p.cos_sin + (int64_t)t * p.rot + (i >> 1);
                    const int half = p.rot >> 1;
                    const float c0 = cs[0], s0 = cs[half];
                    const float e = y.x, f = y.y;
                    y.x = e * c0 - f * s0;
                    y.y = f * c0 + e * s0;
                    if (i + 2 < p.rot) {
                        const float c1 = cs[1], s1 = cs[half + 1];
                        const float m = y.z, o = y.w;
                        y.z = m * c1 - o * s1;
                        y.w = o * c1 + m * s1;
                    }
                }
                dst = kind[k] == 0 ? p.q_out + (int64_t)t * p.ld_q + c : p.k_pages + (((int64_t)page * p.nkv + h) * p.P + pos % p.P) * p.d + i;
            }
            Vec4<T>::store(dst, y);
        }
    }
}

// Any sizes: a block a token, the convolved row in shared memory.
template <typename T>
__global__ void qk_row_norm_kernel(const RowNormParams<T> p) {
    extern __shared__ float row[];                      // [channels]
    __shared__ float2 scratch[32];
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, r = p.token_row[t], pos = p.positions[t];
    const int nqd = p.nq * p.d, nkd = p.nkv * p.d, channels = nqd + nkd + p.nkv * p.dv;
    const int i0 = p.conv_w ? t - p.row_start[r] : 0;
    float* cstate = p.conv_w && p.taps > 1 ? p.state + (int64_t)p.row_slot[r] * p.slot_stride + p.conv_off : nullptr;
    const bool shift = cstate && p.update_single && p.row_start[r + 1] - p.row_start[r] == 1;
    const T* src = p.proj + (int64_t)t * p.ld;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
        const float bias = p.bias ? p.bias[c] : 0.f;
        const float own = to_float(src[c]) + bias;
        float acc = own;
        if (p.conv_w) {
            const float* w = p.conv_w + (int64_t)c * p.taps;
            acc = 0.f;
            for (int j = 0; j < p.taps - 1; ++j) {
                const int idx = i0 - (p.taps - 1) + j;
                const float in = idx >= 0 ? to_float(src[(int64_t)(idx - i0) * p.ld + c]) + bias
                                          : cstate[(int64_t)(p.taps - 1 + idx) * channels + c];
                acc = fmaf(w[j], in, acc);
                if (shift && j > 0) cstate[(int64_t)(j - 1) * channels + c] = in;       // oldest entry first, by the channel's only thread
            }
            if (shift) cstate[(int64_t)(p.taps - 2) * channels + c] = own;
            acc = fmaf(w[p.taps - 1], own, acc);
        }
        row[c] = acc;
        if (c < nqd) sq += acc * acc;
        else if (c < nqd + nkd) sk += acc * acc;
    }
    rown_pair_sum(sq, sk, scratch);                     // (the barrier inside also publishes the row)
    const float inv_q = rsqrtf(sq / p.q_count + p.eps), inv_k = rsqrtf(sk / p.k_count + p.eps);
    const int page = p.block_table[(int64_t)r * p.table_stride + (pos / p.P - p.page_base[r])];
    const int half = p.rot >> 1;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
        if (c >= nqd + nkd) {
            const int h = (c - nqd - nkd) / p.dv, i = (c - nqd - nkd) % p.dv;
            p.v_pages[(((int64_t)page * p.nkv + h) * p.P + pos % p.P) * p.dv + i] = from_float<T>(row[c] * p.v_scale);
            continue;
        }
        const bool is_q = c < nqd;
        const int base = is_q ? 0 : nqd, h = (c - base) / p.d, i = (c - base) % p.d;
        const float* nw = is_q ? p.q_w : p.k_w;
        const float inv = is_q ? inv_q : inv_k;
        auto normed = [&](int e) -> float {             // entry e of this head
            const int cc = base + h * p.d + e;
            return nw ? row[cc] * inv * nw[cc - base] : row[cc];
        };
        float v = normed(i);
        if (i < p.rot) {
            const int pair = p.pairing == 0 ? i % half : i >> 1;
            const bool lo = p.pairing == 0 ? i < half : (i & 1) == 0;
            const int other = p.pairing == 0 ? (lo ? i + half : i - half) : i ^ 1;
            const float cs = p.cos_sin[(int64_t)t * p.rot + pair], sn = p.cos_sin[(int64_t)t * p.rot + half + pair];
            v = lo ? v * cs - normed(other) * sn : v * cs + normed(other) * sn;
        }
        T* dst = is_q ? p.q_out + (int64_t)t * p.ld_q + c : p.k_pages + (((int64_t)page * p.nkv + h) * p.P + pos % p.P) * p.d + i;
        *dst = from_float<T>(v);
    }
}

template <typename T, int TAPS> static int launch_row_norm_vec(const RowNormParams<T>& p, int nvec, cudaStream_t stream) {
    const int tpt = p.tokens > 512 ? 4 : 1;             // a step of few tokens: a block a token
    const int vpt = nvec <= 768 ? 1 : (nvec <= 1024 ? 2 : 4);
    const dim3 grid((p.tokens + tpt - 1) / tpt), block(((nvec + vpt - 1) / vpt + 31) / 32 * 32);
    if (vpt == 1) {
        if (tpt == 1) return acorn_launch(qk_row_norm_vec_kernel<T, TAPS, 1, 1>, grid, block, 0, stream, p);
        return acorn_launch(qk_row_norm_vec_kernel<T, TAPS, 1, 4>, grid, block, 0, stream, p);
    }
    const dim3 one(p.tokens);
    if (vpt == 2) return acorn_launch(qk_row_norm_vec_kernel<T, TAPS, 2, 1>, one, block, 0, stream, p);
    return acorn_launch(qk_row_norm_vec_kernel<T, TAPS, 4, 1>, one, block, 0, stream, p);
}

template <typename T> static int launch_row_norm(const RowNormParams<T>& p, cudaStream_t stream) {
    const int channels = (p.nq + p.nkv) * p.d + p.nkv * p.dv, vec_taps = p.conv_w ? p.taps : 0;
    const uintptr_t all = (uintptr_t)p.proj | (uintptr_t)p.q_out | (uintptr_t)p.k_pages | (uintptr_t)p.v_pages | (uintptr_t)p.q_w |
                          (uintptr_t)p.k_w | (uintptr_t)p.conv_w | (uintptr_t)p.bias | (uintptr_t)p.state;
    if (p.d % 4 == 0 && p.dv % 4 == 0 && vec_taps <= 4 && p.ld % 4 == 0 && p.ld_q % 4 == 0 && p.slot_stride % 4 == 0 &&
        p.conv_off % 4 == 0 && (all & 15) == 0 && (p.rot == 0 || p.pairing == 1) && channels <= 4 * 4 * 512) {
        const int nvec = channels / 4;
        switch (vec_taps) {
            case 0: return launch_row_norm_vec<T, 0>(p, nvec, stream);
            case 1: return launch_row_norm_vec<T, 1>(p, nvec, stream);
            case 2: return launch_row_norm_vec<T, 2>(p, nvec, stream);
            case 3: return launch_row_norm_vec<T, 3>(p, nvec, stream);
            default: return launch_row_norm_vec<T, 4>(p, nvec, stream);
        }
    }
    const size_t smem = (size_t)channels * sizeof(float);
    if (smem > 160 * 1024) return ACORN_ERR_UNSUPPORTED;
    if (smem > 48 * 1024) {
        static AcornPerDevice configured;
        if (!configured.seen()) {
            cudaError_t e = cudaFuncSetAttribute(qk_row_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
            if (e != cudaSuccess) return (int)e;
            configured.mark();
        }
    }
    return acorn_launch(qk_row_norm_kernel<T>, dim3(p.tokens), dim3(256), smem, stream, p);
}

extern "C" int acorn_qk_row_norm(const void* proj, int64_t ld, void* q_out, int64_t ld_q, void* k_pages, void* v_pages,
                                 const float* q_w, const float* k_w, const float* conv_w, int taps, const float* bias,
                                 float* state, int64_t slot_stride, int64_t conv_off, const int* row_start,
                                 const int* row_slot, int update_single, const int* token_row, const int* positions,
                                 const int* block_table, const int* page_base, int table_stride, const float* cos_sin, int tokens,
                                 int nq, int nkv, int d, int dv, int P, int rot, int pairing, int q_count, int k_count, float eps, float v_scale,
                                 int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (nq < 1 || nkv < 1 || d < 1 || dv < 1 || rot < 0 || rot > d || (rot & 1) || (rot && !cos_sin) || q_count < 1 || k_count < 1 ||
        (conv_w && (taps < 1 || taps > ROWN_MAX_TAPS || (taps > 1 && (!state || !row_slot || !row_start)))))
        return ACORN_ERR_UNSUPPORTED;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        RowNormParams<T> p;
        p.proj = (const T*)proj; p.ld = ld; p.q_out = (T*)q_out; p.ld_q = ld_q; p.k_pages = (T*)k_pages; p.v_pages = (T*)v_pages;
        p.q_w = q_w; p.k_w = k_w; p.conv_w = conv_w; p.bias = bias; p.state = state; p.slot_stride = slot_stride;
        p.conv_off = conv_off; p.row_start = row_start; p.row_slot = row_slot; p.token_row = token_row; p.positions = positions;
        p.block_table = block_table; p.page_base = page_base; p.table_stride = table_stride; p.cos_sin = cos_sin;
        p.tokens = tokens; p.nq = nq; p.nkv = nkv; p.d = d; p.dv = dv; p.P = P; p.rot = rot; p.pairing = pairing; p.taps = taps;
        p.update_single = update_single; p.q_count = (float)q_count; p.k_count = (float)k_count; p.eps = eps; p.v_scale = v_scale;
        return launch_row_norm<T>(p, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}
