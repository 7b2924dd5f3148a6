// Two recurrences over chunks of 64 tokens (float32 throughout).
//
// The gated delta rule with one decay per head:
//     S_i = g_i S_(i-1) + k_i u_i^T,   u_i = beta_i (v_i - g_i S_(i-1)^T k_i),   o_i = S_i^T q_i.
// Within a chunk that starts from S_0, with b_i the sum of the log decays up to i and G_ij = exp(b_i - b_j) (at most one for
// j <= i), the u_i solve a unit lower triangular system, so what hangs on S_0 can be split off:
//     (1 + A) U = diag(beta) V - diag(beta exp(b)) K S_0,   A_ij = beta_i G_ij (k_i . k_j) for j < i
//     U = Ubar - W S_0,   O = diag(exp(b)) Q S_0 + P U,   P_ij = G_ij (q_i . k_j) for j <= i
//     S_end = exp(b_n) S_0 + sum_j G_nj k_j u_j^T
// (the form known from Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule").  Three kernels:
//   delta_chunk_solve   all chunks side by side: b, A, P, and W and Ubar by forward substitution, a column a thread
//   delta_chunk_state   a row's chunks one after the other, heads and tiles of 16 value columns side by side: U and the state
//                       every chunk starts from; the row's end state into its slot
//   delta_chunk_out     all chunks side by side: O
//
// Gated linear attention, S_i = diag(a_i) S_(i-1) + k_i v_i^T, o_i = S_i^T q_i, with a decay per key channel: with b_i the sums of
// the logarithms per channel up to i,
//     O = Q' S_0 + P V,   Q'_i = q_i exp(b_i),   P_ij = sum_d q_id k_jd exp(b_id - b_jd) for j <= i
//     S_end = diag(exp(b_n)) S_0 + sum_j (k_j exp(b_n - b_j)) v_j^T
// No exponent is positive: entries of P between two blocks of 16 tokens take the sums at the later block's start as reference,
// those within a block are evaluated one by one.
//   linear_chunk_local  all chunks side by side, from the projected rows: b, Q', P, the chunk's own sum over k v^T, v in float32
//   linear_chunk_fold   per state entry along a row's chunks: the state every chunk starts from, the end state into the slot
//   delta_chunk_out     as above, with Q' and v in place of q and U
//
// A row's chunks are counted from its first token of the step; chunk c of row r is number row_start[r] / 64 + r + c of the
// step (distinct for all chunks; some numbers stay unused).
#include "common.cuh"

#define DC 64                       // tokens a chunk
#define DC_VT 16                    // value columns a block of delta_chunk_state
#define DC_OT 64                    // value columns a block of delta_chunk_out
#define DC_PAD 4                    // floats between rows in shared memory (16-byte reads of neighbouring rows hit distinct banks)

struct DeltaChunkParams {
    const float* q;                 // [T, KH, dim]
    const float* k;
    const float* v;                 // [T, H, vdim]
    const float* beta;              // [T, H]
    const float* log_g;             // [T, H]
    float* state;                   // slots: [H, dim, vdim]
    int64_t slot_stride;
    const int* row_start;
    const int* row_slot;
    float* w;                       // scratch: [T, H, dim]
    float* u;                       // [T, H, vdim]: Ubar, then U
    float* p;                       // [T, H, DC]
    float* b;                       // [T, H]
    float* s0;                      // [chunk numbers, H, dim, vdim]
    float* out;                     // [T, H, vdim]
    int rows, H, KH, dim, vdim;
};

template <typename T> struct LinearChunkParams {
    const T* in;                    // [tokens, ld]: q (H dim), k (H dim), v (H vdim) as projected
    int64_t ld;
    const float* z;                 // [tokens, ldz] the decays' pre-activations (H dim)
    int64_t ldz;
    const float* bias;              // [H dim]
    float inv_tau, q_scale;
    const int* row_start;
    float* q;                       // [T, H, dim]: Q'
    float* v;                       // [T, H, vdim]
    float* p;                       // [T, H, DC]
    float* s0;                      // [chunk numbers, H, dim, vdim]: the chunk's own sum
    float* decay;                   // [chunk numbers, H, dim]
    int rows, H, dim, vdim;
};

// The row and chunk of a chunk number, or false for an unused one.
__device__ __forceinline__ bool chunk_of(int id, const int* __restrict__ row_start, int rows, int& r, int& first, int& n) {
    int lo = 0, hi = rows - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (row_start[mid] / DC + mid <= id) lo = mid;
        else hi = mid - 1;
    }
    r = lo;
    const int start = row_start[lo], c = id - (start / DC + lo);
    first = start + c * DC;
    n = min(DC, row_start[lo + 1] - first);
    return n > 0;
}

__device__ __forceinline__ void dc_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// n rows of `width` floats (a multiple of 4), ld apart, into DC rows of DP + DC_PAD; the rest zeros
template <int DP> __device__ __forceinline__ void load_rows(float* dst, const float* src, int64_t ld, int n, int width) {
    for (int e = threadIdx.x; e < DC * (DP / 4); e += blockDim.x) {
        const int i = e / (DP / 4), c = (e % (DP / 4)) * 4;
        float* d = dst + i * (DP + DC_PAD) + c;
        if (i < n && c < width) dc_cp16(d, src + (int64_t)i * ld + c);
        else *reinterpret_cast<float4*>(d) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
}

__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
    return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, acc))));
}

template <int DP>
__global__ void __launch_bounds__(256, 2) delta_chunk_solve_kernel(const DeltaChunkParams p) {
    constexpr int LD = DP + DC_PAD, LA = DC + DC_PAD;
    extern __shared__ __align__(16) float sm[];
    float* sK = sm;                                     // [DC][LD]
    float* sQ = sK + DC * LD;                           // [DC][LD]
    float* sA = sQ + DC * LD;                           // [DC][LA]
    __shared__ float sb[DC], sbeta[DC];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, kh = h / (p.H / p.KH), tid = threadIdx.x;
    int r, first, n;
    if (!chunk_of(blockIdx.x, p.row_start, p.rows, r, first, n)) return;
    load_rows<DP>(sK, p.k + ((int64_t)first * p.KH + kh) * p.dim, (int64_t)p.KH * p.dim, n, p.dim);
    load_rows<DP>(sQ, p.q + ((int64_t)first * p.KH + kh) * p.dim, (int64_t)p.KH * p.dim, n, p.dim);
    asm volatile("cp.async.commit_group;\n" ::);
    if (tid < 32) {                                     // sums of the log decays: two tokens a lane
        const int i = 2 * tid;
        const float a = i < n ? p.log_g[(int64_t)(first + i) * p.H + h] : 0.f;
        const float c = i + 1 < n ? p.log_g[(int64_t)(first + i + 1) * p.H + h] : 0.f;
        float run = a + c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float before = __shfl_up_sync(0xffffffffu, run, o);
            if (tid >= o) run += before;
        }
        sb[i] = run - c;
        sb[i + 1] = run;
        if (i < n) p.b[(int64_t)(first + i) * p.H + h] = run - c;
        if (i + 1 < n) p.b[(int64_t)(first + i + 1) * p.H + h] = run;
    } else if (tid < 32 + DC) {
        const int i = tid - 32;
        sbeta[i] = i < n ? p.beta[(int64_t)(first + i) * p.H + h] : 0.f;
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    // k . k and q . k of rows ty + 16 ii and columns tx + 16 jj, the blocks on and below the diagonal
    const int tx = tid & 15, ty = tid >> 4;
    float kk[4][4], qk[4][4];
#pragma unroll
    for (int ii = 0; ii < 4; ++ii)
#pragma unroll
        for (int jj = 0; jj < 4; ++jj) kk[ii][jj] = qk[ii][jj] = 0.f;
#pragma unroll 2
    for (int d = 0; d < DP; d += 4) {
        float4 kj[4];
#pragma unroll
        for (int jj = 0; jj < 4; ++jj) kj[jj] = *reinterpret_cast<const float4*>(sK + (tx + 16 * jj) * LD + d);
#pragma unroll
        for (int ii = 0; ii < 4; ++ii) {
            const float4 ki = *reinterpret_cast<const float4*>(sK + (ty + 16 * ii) * LD + d);
            const float4 qi = *reinterpret_cast<const float4*>(sQ + (ty + 16 * ii) * LD + d);
#pragma unroll
            for (int jj = 0; jj <= ii; ++jj) {
                kk[ii][jj] = dot4(ki, kj[jj], kk[ii][jj]);
                qk[ii][jj] = dot4(qi, kj[jj], qk[ii][jj]);
            }
        }
    }
#pragma unroll
    for (int ii = 0; ii < 4; ++ii) {
        const int i = ty + 16 * ii;
#pragma unroll
        for (int jj = 0; jj <= ii; ++jj) {
            const int j = tx + 16 * jj;
            const float G = j <= i ? expf(sb[i] - sb[j]) : 0.f;
            sA[i * LA + j] = j < i ? sbeta[i] * G * kk[ii][jj] : 0.f;
            if (i < n) p.p[((int64_t)(first + i) * p.H + h) * DC + j] = G * qk[ii][jj];
        }
    }
    __syncthreads();
    // forward substitution: a thread a column of [W | Ubar], its 64 entries in registers
    for (int c0 = 0; c0 < p.dim + p.vdim; c0 += 256) {
        const int col = c0 + tid;
        if (col >= p.dim + p.vdim) break;
        const bool is_w = col < p.dim;
        float x[DC];
        if (is_w) {
#pragma unroll
            for (int i = 0; i < DC; ++i) x[i] = sbeta[i] * expf(sb[i]) * sK[i * LD + col];
        } else {
            const float* v = p.v + ((int64_t)first * p.H + h) * p.vdim + col - p.dim;
#pragma unroll
            for (int i = 0; i < DC; ++i) x[i] = i < n ? v[(int64_t)i * p.H * p.vdim] : 0.f;
#pragma unroll
            for (int i = 0; i < DC; ++i) x[i] *= sbeta[i];
        }
#pragma unroll
        for (int i = 1; i < DC; ++i) {
            float s0 = 0.f, s1 = 0.f;
#pragma unroll
            for (int j = 0; j < i; j += 4) {            // entries from j = i on are zeros in A
                const float4 a = *reinterpret_cast<const float4*>(sA + i * LA + j);
                s0 = fmaf(a.x, x[j], s0);
                if (j + 1 < i) s1 = fmaf(a.y, x[j + 1], s1);
                if (j + 2 < i) s0 = fmaf(a.z, x[j + 2], s0);
                if (j + 3 < i) s1 = fmaf(a.w, x[j + 3], s1);
            }
            x[i] -= s0 + s1;
        }
        float* dst = is_w ? p.w + ((int64_t)first * p.H + h) * p.dim + col : p.u + ((int64_t)first * p.H + h) * p.vdim + col - p.dim;
        const int64_t ld = (int64_t)p.H * (is_w ? p.dim : p.vdim);
#pragma unroll
        for (int i = 0; i < DC; ++i)
            if (i < n) dst[i * ld] = x[i];
    }
}

// Both products of a chunk have few outputs (64 x 16 and dim x 16) and a long sum, so a warp takes a slice of the sum for large
// register tiles (8 x 4 a lane: three reads of shared memory for 32 multiply-adds) and the slices are added up through
// shared memory: U over 8 slices of the key channels, the state over 4 slices of the tokens by 2 halves of the channels.
template <int DP>
__global__ void __launch_bounds__(256) delta_chunk_state_kernel(const DeltaChunkParams p) {
    constexpr int LD = DP + DC_PAD, LV = DC_VT + DC_PAD, SLICE = DP / 8, ND = DP / 64 > 0 ? DP / 64 : 1;
    constexpr int PARTS = 8 * DC > 4 * DP ? 8 * DC : 4 * DP;
    extern __shared__ __align__(16) float sm[];
    float* sW = sm;                                     // [2][DC][LD]
    float* sK = sW + 2 * DC * LD;                       // [2][DC][LD]
    float* sS = sK + 2 * DC * LD;                       // [DP][LV] the state's tile
    float* sU = sS + DP * LV;                           // [DC][LV] a token's u times G_nj
    float* part = sU + DC * LV;                         // [PARTS][LV] slices of the sums
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, r = blockIdx.z, kh = h / (p.H / p.KH), v0 = blockIdx.x * DC_VT, tid = threadIdx.x;
    const int lane = tid & 31, warp = tid >> 5, rg = lane >> 2, cg = lane & 3;
    const int start = p.row_start[r], L = p.row_start[r + 1] - start;
    const int chunks = (L + DC - 1) / DC, id0 = start / DC + r;
    const int c4 = v0 + 4 * (tid & 3);                  // this thread's four columns when sums are collected
    const bool on = c4 < p.vdim;
    float* slot = p.state + (int64_t)p.row_slot[r] * p.slot_stride + (int64_t)h * p.dim * p.vdim;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    // the state entries this thread keeps: key channels (tid + 256 m) / 4, columns c4 ..
    float4 S[ND];
#pragma unroll
    for (int m = 0; m < ND; ++m) {
        const int d = (tid + 256 * m) >> 2;
        S[m] = zero;
        if (d < p.dim && on) {                          // (a slot starts wherever it may: no vector reads)
            const float* at = slot + (int64_t)d * p.vdim + c4;
            S[m] = make_float4(at[0], at[1], at[2], at[3]);
        }
    }
    auto publish = [&]() {
#pragma unroll
        for (int m = 0; m < ND; ++m) {
            const int d = (tid + 256 * m) >> 2;
            if (d < DP) *reinterpret_cast<float4*>(sS + d * LV + 4 * (tid & 3)) = S[m];
        }
    };
    publish();
    auto fetch = [&](int c) {
        const int first = start + c * DC, n = min(DC, L - c * DC);
        load_rows<DP>(sW + (c & 1) * DC * LD, p.w + ((int64_t)first * p.H + h) * p.dim, (int64_t)p.H * p.dim, n, p.dim);
        load_rows<DP>(sK + (c & 1) * DC * LD, p.k + ((int64_t)first * p.KH + kh) * p.dim, (int64_t)p.KH * p.dim, n, p.dim);
    };
    auto axpy = [](float a, const float4& x, float4& y) {
        y.x = fmaf(a, x.x, y.x); y.y = fmaf(a, x.y, y.y); y.z = fmaf(a, x.z, y.z); y.w = fmaf(a, x.w, y.w);
    };
    auto add = [](float4& y, const float4& x) { y.x += x.x; y.y += x.y; y.z += x.z; y.w += x.w; };
    if (chunks > 0) fetch(0);
    asm volatile("cp.async.commit_group;\n" ::);
    const int token = tid >> 2;                         // the token whose u this thread collects
    for (int c = 0; c < chunks; ++c) {
        const int first = start + c * DC, n = min(DC, L - c * DC);
        const float bn = p.b[(int64_t)(first + n - 1) * p.H + h];
        const int64_t t = (int64_t)(first + min(token, n - 1)) * p.H + h;
        const bool live = token < n && on;
        const float4 ub = live ? *reinterpret_cast<const float4*>(p.u + t * p.vdim + c4) : zero;
        const float bj = p.b[t];
        if (c + 1 < chunks) fetch(c + 1);
        asm volatile("cp.async.commit_group;\n" ::);
        float* keep = p.s0 + ((int64_t)(id0 + c) * p.H + h) * p.dim * p.vdim;      // the state this chunk starts from
#pragma unroll
        for (int m = 0; m < ND; ++m) {
            const int d = (tid + 256 * m) >> 2;
            if (d < p.dim && on) *reinterpret_cast<float4*>(keep + (int64_t)d * p.vdim + c4) = S[m];
        }
        asm volatile("cp.async.wait_group 1;\n" ::);
        __syncthreads();                                // this chunk's rows and the state's tile are there
        {
            const float* W = sW + (c & 1) * DC * LD + warp * SLICE;
            float4 acc[8];
#pragma unroll
            for (int rr = 0; rr < 8; ++rr) acc[rr] = zero;
#pragma unroll
            for (int d = 0; d < SLICE; d += 4) {
                float4 s[4];
#pragma unroll
                for (int q = 0; q < 4; ++q) s[q] = *reinterpret_cast<const float4*>(sS + (warp * SLICE + d + q) * LV + 4 * cg);
#pragma unroll
                for (int rr = 0; rr < 8; ++rr) {
                    const float4 w = *reinterpret_cast<const float4*>(W + (rg + 8 * rr) * LD + d);
                    axpy(w.x, s[0], acc[rr]); axpy(w.y, s[1], acc[rr]); axpy(w.z, s[2], acc[rr]); axpy(w.w, s[3], acc[rr]);
                }
            }
#pragma unroll
            for (int rr = 0; rr < 8; ++rr) *reinterpret_cast<float4*>(part + (warp * DC + rg + 8 * rr) * LV + 4 * cg) = acc[rr];
        }
        __syncthreads();
        {
            float4 u = zero;
#pragma unroll
            for (int q = 0; q < 8; ++q) add(u, *reinterpret_cast<const float4*>(part + (q * DC + token) * LV + 4 * (tid & 3)));
            u = make_float4(ub.x - u.x, ub.y - u.y, ub.z - u.z, ub.w - u.w);
            if (live) *reinterpret_cast<float4*>(p.u + t * p.vdim + c4) = u;
            const float G = token < n ? expf(bn - bj) : 0.f;
            *reinterpret_cast<float4*>(sU + token * LV + 4 * (tid & 3)) = make_float4(u.x * G, u.y * G, u.z * G, u.w * G);
        }
        __syncthreads();
        {
            const int jg = warp >> 1, d0 = (warp & 1) * (DP / 2) + 4 * rg;         // key channels d0 + 32 m .. + 3
            if (4 * rg < DP / 2) {
                const float* K = sK + (c & 1) * DC * LD + jg * 16 * LD + d0;
                float4 acc[ND][4];
#pragma unroll
                for (int m = 0; m < ND; ++m)
#pragma unroll
                    for (int q = 0; q < 4; ++q) acc[m][q] = zero;
#pragma unroll 8
                for (int j = 0; j < 16; ++j) {
                    const float4 u = *reinterpret_cast<const float4*>(sU + (jg * 16 + j) * LV + 4 * cg);
#pragma unroll
                    for (int m = 0; m < ND; ++m) {
                        const float4 k = *reinterpret_cast<const float4*>(K + j * LD + 32 * m);
                        axpy(k.x, u, acc[m][0]); axpy(k.y, u, acc[m][1]); axpy(k.z, u, acc[m][2]); axpy(k.w, u, acc[m][3]);
                    }
                }
#pragma unroll
                for (int m = 0; m < ND; ++m)
#pragma unroll
                    for (int q = 0; q < 4; ++q) *reinterpret_cast<float4*>(part + (jg * DP + d0 + 32 * m + q) * LV + 4 * cg) = acc[m][q];
            }
        }
        __syncthreads();
        const float gn = expf(bn);
#pragma unroll
        for (int m = 0; m < ND; ++m) {
            const int d = (tid + 256 * m) >> 2;
            if (d >= DP) break;
            S[m] = make_float4(S[m].x * gn, S[m].y * gn, S[m].z * gn, S[m].w * gn);
#pragma unroll
            for (int q = 0; q < 4; ++q) add(S[m], *reinterpret_cast<const float4*>(part + (q * DP + d) * LV + 4 * (tid & 3)));
        }
        publish();
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
#pragma unroll
    for (int m = 0; m < ND; ++m) {
        const int d = (tid + 256 * m) >> 2;
        if (d < p.dim && on) {
            float* at = slot + (int64_t)d * p.vdim + c4;
            at[0] = S[m].x; at[1] = S[m].y; at[2] = S[m].z; at[3] = S[m].w;
        }
    }
}

// SCALED: q already holds exp(b) (and b is not read)
template <int DP, bool SCALED>
__global__ void __launch_bounds__(256, 2) delta_chunk_out_kernel(const DeltaChunkParams p) {
    constexpr int LD = DP + DC_PAD, LO = DC_OT + DC_PAD, LA = DC + DC_PAD;
    extern __shared__ __align__(16) float sm[];
    float* sQ = sm;                                     // [DC][LD]
    float* sS = sQ + DC * LD;                           // [DP][LO]
    float* sU = sS + DP * LO;                           // [DC][LO]
    float* sP = sU + DC * LO;                           // [DC][LA]
    __shared__ float sb[DC];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, kh = h / (p.H / p.KH), v0 = blockIdx.z * DC_OT, tid = threadIdx.x;
    int r, first, n;
    if (!chunk_of(blockIdx.x, p.row_start, p.rows, r, first, n)) return;
    load_rows<DP>(sQ, p.q + ((int64_t)first * p.KH + kh) * p.dim, (int64_t)p.KH * p.dim, n, p.dim);
    const float* S = p.s0 + ((int64_t)blockIdx.x * p.H + h) * p.dim * p.vdim + v0;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int e = tid; e < DP * (DC_OT / 4); e += 256) {
        const int d = e / (DC_OT / 4), c = (e % (DC_OT / 4)) * 4;
        if (d < p.dim && v0 + c < p.vdim) dc_cp16(sS + d * LO + c, S + (int64_t)d * p.vdim + c);
        else *reinterpret_cast<float4*>(sS + d * LO + c) = zero;
    }
    for (int e = tid; e < DC * (DC_OT / 4); e += 256) {
        const int j = e / (DC_OT / 4), c = (e % (DC_OT / 4)) * 4;
        if (j < n && v0 + c < p.vdim) dc_cp16(sU + j * LO + c, p.u + ((int64_t)(first + j) * p.H + h) * p.vdim + v0 + c);
        else *reinterpret_cast<float4*>(sU + j * LO + c) = zero;
    }
    for (int e = tid; e < DC * (DC / 4); e += 256) {
        const int i = e / (DC / 4), j = (e % (DC / 4)) * 4;
        if (i < n && j / 16 <= i / 16) dc_cp16(sP + i * LA + j, p.p + ((int64_t)(first + i) * p.H + h) * DC + j);
        else *reinterpret_cast<float4*>(sP + i * LA + j) = zero;
    }
    asm volatile("cp.async.commit_group;\n" ::);
    if (!SCALED && tid < DC) sb[tid] = p.b[(int64_t)(first + min(tid, n - 1)) * p.H + h];
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    const int tx = tid & 15, ty = tid >> 4;             // rows ty + 16 ii, columns 4 tx .. 4 tx + 3
    float4 acc[4];
#pragma unroll
    for (int ii = 0; ii < 4; ++ii) acc[ii] = zero;
    auto axpy = [](float a, const float4& x, float4& y) {
        y.x = fmaf(a, x.x, y.x); y.y = fmaf(a, x.y, y.y); y.z = fmaf(a, x.z, y.z); y.w = fmaf(a, x.w, y.w);
    };
#pragma unroll 2
    for (int d = 0; d < DP; d += 4) {
        float4 s[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) s[q] = *reinterpret_cast<const float4*>(sS + (d + q) * LO + 4 * tx);
#pragma unroll
        for (int ii = 0; ii < 4; ++ii) {
            const float4 q4 = *reinterpret_cast<const float4*>(sQ + (ty + 16 * ii) * LD + d);
            axpy(q4.x, s[0], acc[ii]); axpy(q4.y, s[1], acc[ii]); axpy(q4.z, s[2], acc[ii]); axpy(q4.w, s[3], acc[ii]);
        }
    }
    if (!SCALED) {
#pragma unroll
        for (int ii = 0; ii < 4; ++ii) {
            const float g = expf(sb[ty + 16 * ii]);
            acc[ii] = make_float4(acc[ii].x * g, acc[ii].y * g, acc[ii].z * g, acc[ii].w * g);
        }
    }
#pragma unroll
    for (int jb = 0; jb < 4; ++jb) {                    // blocks of 16 keys; rows before the block see none of it
#pragma unroll
        for (int j = 16 * jb; j < 16 * jb + 16; j += 4) {
            float4 u[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) u[q] = *reinterpret_cast<const float4*>(sU + (j + q) * LO + 4 * tx);
#pragma unroll
            for (int ii = jb; ii < 4; ++ii) {
                const float4 p4 = *reinterpret_cast<const float4*>(sP + (ty + 16 * ii) * LA + j);
                axpy(p4.x, u[0], acc[ii]); axpy(p4.y, u[1], acc[ii]); axpy(p4.z, u[2], acc[ii]); axpy(p4.w, u[3], acc[ii]);
            }
        }
    }
#pragma unroll
    for (int ii = 0; ii < 4; ++ii) {
        const int i = ty + 16 * ii;
        if (i < n && v0 + 4 * tx < p.vdim)
            *reinterpret_cast<float4*>(p.out + ((int64_t)(first + i) * p.H + h) * p.vdim + v0 + 4 * tx) = acc[ii];
    }
}

template <int DP> static int launch_delta_chunk(const DeltaChunkParams& p, int ids, cudaStream_t stream) {
    constexpr int LD = DP + DC_PAD;
    const size_t solve = (size_t)(2 * DC * LD + DC * (DC + DC_PAD)) * sizeof(float);
    constexpr int LV = DC_VT + DC_PAD, PARTS = 8 * DC > 4 * DP ? 8 * DC : 4 * DP;
    const size_t walk = (size_t)(4 * DC * LD + (DP + DC + PARTS) * LV) * sizeof(float);
    const size_t out = (size_t)(DC * LD + DP * (DC_OT + DC_PAD) + DC * (DC_OT + DC_PAD) + DC * (DC + DC_PAD)) * sizeof(float);
    static AcornPerDevice configured;
    if (!configured.seen()) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_solve_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)solve);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_state_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)walk);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_out_kernel<DP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out);
        if (e != cudaSuccess) return (int)e;
        configured.mark();
    }
    int rc = acorn_launch(delta_chunk_solve_kernel<DP>, dim3(ids, p.H), dim3(256), solve, stream, p);
    if (rc) return rc;
    rc = acorn_launch(delta_chunk_state_kernel<DP>, dim3((p.vdim + DC_VT - 1) / DC_VT, p.H, p.rows), dim3(256), walk, stream, p);
    if (rc) return rc;
    return acorn_launch(delta_chunk_out_kernel<DP, false>, dim3(ids, p.H, (p.vdim + DC_OT - 1) / DC_OT), dim3(256), out, stream, p);
}

// ---------------------------------------------------------------- gated linear attention

__device__ __forceinline__ float dc_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

template <typename T, int DP>
__global__ void __launch_bounds__(256) linear_chunk_local_kernel(const LinearChunkParams<T> p) {
    constexpr int LD = DP + DC_PAD, LO = DC_OT + DC_PAD, DQ = DP / 4;
    extern __shared__ __align__(16) float sm[];
    float* sQ = sm;                                     // [DC][LD]
    float* sK = sQ + DC * LD;                           // [DC][LD]
    float* sB = sK + DC * LD;                           // [DC][LD] sums of the logarithms (to base 2)
    float* sR = sB + DC * LD;                           // [48][LD] keys of the blocks before one, at its reference
    float* sV = sR + 48 * LD;                           // [DC][LO]
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, tid = threadIdx.x;
    int r, first, n;
    if (!chunk_of(blockIdx.x, p.row_start, p.rows, r, first, n)) return;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const int Hd = p.H * p.dim;
    const float to_log2 = -1.4426950408889634f * p.inv_tau;
    for (int e = tid; e < DC * DQ; e += 256) {
        const int i = e / DQ, c = (e % DQ) * 4, at = i * LD + c;
        float4 q = zero, k = zero, l = zero;
        if (i < n && c < p.dim) {
            const T* row = p.in + (int64_t)(first + i) * p.ld + h * p.dim + c;
            q = Vec4<T>::load(row);
            k = Vec4<T>::load(row + Hd);
            const float4 z = *reinterpret_cast<const float4*>(p.z + (int64_t)(first + i) * p.ldz + h * p.dim + c);
            const float4 b = *reinterpret_cast<const float4*>(p.bias + h * p.dim + c);
            q = make_float4(q.x * p.q_scale, q.y * p.q_scale, q.z * p.q_scale, q.w * p.q_scale);
            l = make_float4(dc_softplus(-(z.x + b.x)) * to_log2, dc_softplus(-(z.y + b.y)) * to_log2,
                            dc_softplus(-(z.z + b.z)) * to_log2, dc_softplus(-(z.w + b.w)) * to_log2);
        }
        *reinterpret_cast<float4*>(sQ + at) = q;
        *reinterpret_cast<float4*>(sK + at) = k;
        *reinterpret_cast<float4*>(sB + at) = l;
    }
    __syncthreads();
    for (int e = tid; e < 4 * DP; e += 256) {           // sums within blocks of 16 tokens, then over the blocks before
        float run = 0.f;
        float* col = sB + (e / DP) * 16 * LD + e % DP;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            run += col[i * LD];
            col[i * LD] = run;
        }
    }
    __syncthreads();
    float before[(4 * DP + 255) / 256];
#pragma unroll
    for (int m = 0; m < (4 * DP + 255) / 256; ++m) {
        const int e = tid + 256 * m;
        before[m] = 0.f;
        if (e < 4 * DP)
            for (int s = 0; s < e / DP; ++s) before[m] += sB[(16 * s + 15) * LD + e % DP];
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < (4 * DP + 255) / 256; ++m) {
        const int e = tid + 256 * m;
        if (e < 4 * DP && e >= DP)
#pragma unroll
            for (int i = 0; i < 16; ++i) sB[((e / DP) * 16 + i) * LD + e % DP] += before[m];
    }
    __syncthreads();
    auto exp4 = [](const float4& a, const float4& b) -> float4 {       // 2^(a - b)
        return make_float4(exp2f(a.x - b.x), exp2f(a.y - b.y), exp2f(a.z - b.z), exp2f(a.w - b.w));
    };
    auto mul4 = [](const float4& a, const float4& b) -> float4 { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); };
    // entries within blocks of 16 tokens
    const int tx = tid & 15, ty = tid >> 4;
    float* P = p.p + ((int64_t)first * p.H + h) * DC;
    const int64_t ldp = (int64_t)p.H * DC;
#pragma unroll
    for (int I = 0; I < 4; ++I) {
        const int i = 16 * I + ty, j = 16 * I + tx;
        float s = 0.f;
        if (tx <= ty) {
#pragma unroll 4
            for (int d = 0; d < DP; d += 4) {
                const float4 q = *reinterpret_cast<const float4*>(sQ + i * LD + d), k = *reinterpret_cast<const float4*>(sK + j * LD + d);
                const float4 bi = *reinterpret_cast<const float4*>(sB + i * LD + d), bj = *reinterpret_cast<const float4*>(sB + j * LD + d);
                s = dot4(mul4(q, k), exp4(bi, bj), s);
            }
        }
        if (i < n) P[i * ldp + j] = s;
    }
    __syncthreads();
    // Q' to memory; in shared memory q at its block's reference
    for (int e = tid; e < DC * DQ; e += 256) {
        const int i = e / DQ, c = (e % DQ) * 4, at = i * LD + c;
        const float4 q = *reinterpret_cast<const float4*>(sQ + at), b = *reinterpret_cast<const float4*>(sB + at);
        if (i < n && c < p.dim) *reinterpret_cast<float4*>(p.q + ((int64_t)(first + i) * p.H + h) * p.dim + c) = mul4(q, exp4(b, zero));
        if (i >= 16) *reinterpret_cast<float4*>(sQ + at) = mul4(q, exp4(b, *reinterpret_cast<const float4*>(sB + ((i & ~15) - 1) * LD + c)));
    }
    if (tid < DQ && 4 * tid < p.dim)
        *reinterpret_cast<float4*>(p.decay + ((int64_t)blockIdx.x * p.H + h) * p.dim + 4 * tid) =
            exp4(*reinterpret_cast<const float4*>(sB + (DC - 1) * LD + 4 * tid), zero);
#pragma unroll
    for (int I = 1; I < 4; ++I) {                       // entries against the blocks before
        for (int e = tid; e < 16 * I * DQ; e += 256) {
            const int j = e / DQ, c = (e % DQ) * 4;
            *reinterpret_cast<float4*>(sR + j * LD + c) =
                mul4(*reinterpret_cast<const float4*>(sK + j * LD + c),
                     exp4(*reinterpret_cast<const float4*>(sB + (16 * I - 1) * LD + c), *reinterpret_cast<const float4*>(sB + j * LD + c)));
        }
        __syncthreads();
        const int i = 16 * I + ty;
        float s[3] = {0.f, 0.f, 0.f};
#pragma unroll 4
        for (int d = 0; d < DP; d += 4) {
            const float4 q = *reinterpret_cast<const float4*>(sQ + i * LD + d);
#pragma unroll
            for (int J = 0; J < I; ++J) s[J] = dot4(q, *reinterpret_cast<const float4*>(sR + (16 * J + tx) * LD + d), s[J]);
        }
        if (i < n)
#pragma unroll
            for (int J = 0; J < I; ++J) P[i * ldp + 16 * J + tx] = s[J];
        __syncthreads();
    }
    // the keys at the chunk's end, and their sum with the values
    for (int e = tid; e < DC * DQ; e += 256) {
        const int at = (e / DQ) * LD + (e % DQ) * 4;
        *reinterpret_cast<float4*>(sK + at) = mul4(*reinterpret_cast<const float4*>(sK + at),
                                                   exp4(*reinterpret_cast<const float4*>(sB + (DC - 1) * LD + (e % DQ) * 4),
                                                        *reinterpret_cast<const float4*>(sB + at)));
    }
    constexpr int ND = DP / 64 > 0 ? DP / 64 : 1;       // groups of 4 key channels a thread
    for (int v0 = 0; v0 < p.vdim; v0 += DC_OT) {
        for (int e = tid; e < DC * (DC_OT / 4); e += 256) {
            const int j = e / (DC_OT / 4), c = (e % (DC_OT / 4)) * 4;
            float4 v = zero;
            if (j < n && v0 + c < p.vdim) {
                v = Vec4<T>::load(p.in + (int64_t)(first + j) * p.ld + 2 * Hd + h * p.vdim + v0 + c);
                *reinterpret_cast<float4*>(p.v + ((int64_t)(first + j) * p.H + h) * p.vdim + v0 + c) = v;
            }
            *reinterpret_cast<float4*>(sV + j * LO + c) = v;
        }
        __syncthreads();
        float4 acc[ND][4];
#pragma unroll
        for (int m = 0; m < ND; ++m)
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[m][q] = zero;
        if (4 * ty < DP) {
#pragma unroll 4
            for (int j = 0; j < DC; ++j) {
                const float4 v = *reinterpret_cast<const float4*>(sV + j * LO + 4 * tx);
#pragma unroll
                for (int m = 0; m < ND; ++m) {
                    const float4 k = *reinterpret_cast<const float4*>(sK + j * LD + 4 * ty + 64 * m);
                    const float kk[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        acc[m][q].x = fmaf(kk[q], v.x, acc[m][q].x); acc[m][q].y = fmaf(kk[q], v.y, acc[m][q].y);
                        acc[m][q].z = fmaf(kk[q], v.z, acc[m][q].z); acc[m][q].w = fmaf(kk[q], v.w, acc[m][q].w);
                    }
                }
            }
            float* E = p.s0 + ((int64_t)blockIdx.x * p.H + h) * p.dim * p.vdim;
#pragma unroll
            for (int m = 0; m < ND; ++m)
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const int d = 4 * ty + 64 * m + q;
                    if (d < p.dim && v0 + 4 * tx < p.vdim) *reinterpret_cast<float4*>(E + (int64_t)d * p.vdim + v0 + 4 * tx) = acc[m][q];
                }
        }
        __syncthreads();
    }
}

// A thread four value columns of a key channel's state, along a row's chunks; the chunks' sums are fetched a few ahead.
__global__ void linear_chunk_fold_kernel(float* __restrict__ state, int64_t slot_stride, const int* __restrict__ row_start,
                                         const int* __restrict__ row_slot, float* __restrict__ s0, const float* __restrict__ decay,
                                         int H, int dim, int vdim) {
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.z, h = blockIdx.y;
    const int per = dim * (vdim / 4), e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= per) return;
    const int d = e / (vdim / 4);
    const int start = row_start[r], chunks = (row_start[r + 1] - start + DC - 1) / DC, id0 = start / DC + r;
    float4* slot = reinterpret_cast<float4*>(state + (int64_t)row_slot[r] * slot_stride + (int64_t)h * dim * vdim) + e;
    float4* E = reinterpret_cast<float4*>(s0 + ((int64_t)id0 * H + h) * dim * vdim) + e;
    const float* a = decay + ((int64_t)id0 * H + h) * dim + d;
    const int64_t step = (int64_t)H * dim * vdim / 4;
    float4 cur = *slot;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float4 x[AHEAD];
        float f[AHEAD];
#pragma unroll
        for (int q = 0; q < AHEAD; ++q) {
            const int c = min(c0 + q, chunks - 1);
            x[q] = E[c * step];
            f[q] = a[(int64_t)c * H * dim];
        }
#pragma unroll
        for (int q = 0; q < AHEAD; ++q) {
            if (c0 + q >= chunks) break;
            E[(c0 + q) * step] = cur;
            cur = make_float4(fmaf(f[q], cur.x, x[q].x), fmaf(f[q], cur.y, x[q].y), fmaf(f[q], cur.z, x[q].z), fmaf(f[q], cur.w, x[q].w));
        }
    }
    *slot = cur;
}

template <typename T, int DP> static int launch_linear_chunk(const LinearChunkParams<T>& p, const DeltaChunkParams& o, int ids, cudaStream_t stream) {
    constexpr int LD = DP + DC_PAD, LO = DC_OT + DC_PAD;
    const size_t local = (size_t)(3 * DC * LD + 48 * LD + DC * LO) * sizeof(float);
    const size_t out = (size_t)(DC * LD + DP * LO + DC * LO + DC * (DC + DC_PAD)) * sizeof(float);
    static AcornPerDevice configured;
    if (!configured.seen()) {
        cudaError_t e = cudaFuncSetAttribute(linear_chunk_local_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_out_kernel<DP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out);
        if (e != cudaSuccess) return (int)e;
        configured.mark();
    }
    int rc = acorn_launch(linear_chunk_local_kernel<T, DP>, dim3(ids, p.H), dim3(256), local, stream, p);
    if (rc) return rc;
    rc = acorn_launch(linear_chunk_fold_kernel, dim3((p.dim * (p.vdim / 4) + 255) / 256, p.H, p.rows), dim3(256), 0, stream, o.state,
                      o.slot_stride, o.row_start, o.row_slot, p.s0, (const float*)p.decay, p.H, p.dim, p.vdim);
    if (rc) return rc;
    return acorn_launch(delta_chunk_out_kernel<DP, true>, dim3(ids, p.H, (p.vdim + DC_OT - 1) / DC_OT), dim3(256), out, stream, o);
}

extern "C" int acorn_linear_chunk(const void* in, int64_t ld, const float* z, int64_t ldz, const float* bias, float inv_tau, float* state,
                                  int64_t slot_stride, const int* row_start, const int* row_slot, float* q, float* v, float* pp, float* s0,
                                  float* decay, float* out, int tokens, int rows, int H, int dim, int vdim, int dtype, cudaStream_t stream) {
    if (tokens <= 0 || rows <= 0) return 0;
    const uintptr_t all = (uintptr_t)z | (uintptr_t)bias | (uintptr_t)q | (uintptr_t)v | (uintptr_t)s0 | (uintptr_t)out | (uintptr_t)state | (uintptr_t)decay;
    if (dim < 4 || dim > 128 || dim % 4 || vdim < 4 || vdim % 4 || H < 1 || H > 65535 || rows > 65535 || (all & 15) || ld % 4 || ldz % 4 ||
        slot_stride % 4 || ((uintptr_t)in & (dtype == ACORN_DTYPE_BF16 ? 7 : 15)))
        return ACORN_ERR_UNSUPPORTED;
    const DeltaChunkParams o = {q, nullptr, nullptr, nullptr, nullptr, state, slot_stride, row_start, row_slot, nullptr, v, pp, nullptr, s0, out,
                                rows, H, H, dim, vdim};
    const int ids = tokens / DC + rows;
    ACORN_DISPATCH_DTYPE(dtype, T, {
        LinearChunkParams<T> p;
        p.in = (const T*)in; p.ld = ld; p.z = z; p.ldz = ldz; p.bias = bias; p.inv_tau = inv_tau; p.q_scale = (float)(1.0 / sqrt((double)dim));
        p.row_start = row_start; p.q = q; p.v = v; p.p = pp; p.s0 = s0; p.decay = decay; p.rows = rows; p.H = H; p.dim = dim; p.vdim = vdim;
        if (dim <= 32) return launch_linear_chunk<T, 32>(p, o, ids, stream);
        if (dim <= 64) return launch_linear_chunk<T, 64>(p, o, ids, stream);
        return launch_linear_chunk<T, 128>(p, o, ids, stream);
    });
    return ACORN_ERR_UNSUPPORTED;
}

extern "C" int acorn_delta_chunk_supported(int dim, int vdim) { return dim >= 4 && dim <= 128 && dim % 4 == 0 && vdim >= 4 && vdim % 4 == 0; }

// chunk numbers of a step (what s0 must have room for)
extern "C" int acorn_delta_chunk_ids(int tokens, int rows) { return tokens / DC + rows; }

extern "C" int acorn_delta_chunk(const float* q, const float* k, const float* v, const float* beta, const float* log_g, float* state,
                                 int64_t slot_stride, const int* row_start, const int* row_slot, float* w, float* u, float* pp, float* b,
                                 float* s0, float* out, int tokens, int rows, int H, int KH, int dim, int vdim, cudaStream_t stream) {
    if (tokens <= 0 || rows <= 0) return 0;
    const uintptr_t all = (uintptr_t)q | (uintptr_t)k | (uintptr_t)w | (uintptr_t)u | (uintptr_t)pp | (uintptr_t)s0 | (uintptr_t)out;
    if (!acorn_delta_chunk_supported(dim, vdim) || KH < 1 || H < 1 || H % KH || H > 65535 || rows > 65535 || (all & 15)) return ACORN_ERR_UNSUPPORTED;
    DeltaChunkParams p = {q, k, v, beta, log_g, state, slot_stride, row_start, row_slot, w, u, pp, b, s0, out, rows, H, KH, dim, vdim};
    const int ids = acorn_delta_chunk_ids(tokens, rows);
    if (dim <= 32) return launch_delta_chunk<32>(p, ids, stream);
    if (dim <= 64) return launch_delta_chunk<64>(p, ids, stream);
    return launch_delta_chunk<128>(p, ids, stream);
}
