// The gated delta rule: a recurrent mixer whose state is corrected towards each token's value.
//
// Per value head h (query/key head h / (heads / kv_heads)), with a state S [d, dv] that starts at zero:
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
//   delta_prepare   from the 32-bit projection row [q heads | k heads | v heads | ... | b | a ...]: a causal
//                   convolution over time on every channel of q, k and v (the last taps - 1 rows a
//                   sequence has seen are its state, oldest first) and silu; query and key heads divided
//                   by sqrt(sum(x^2) + eps), queries also times d^(-1/2); per value head
//                   beta = sigmoid(b) and the logarithm of the decay, -exp(A_log) softplus(a + dt_bias).
//                   In a step of one token a sequence the same launch moves the convolution's state on.
//   delta_step      one token a sequence: the recurrence with the state read once and written once, and
//                   the output's norm and gate behind it, a block a (head, sequence).
//   delta_scan      several tokens a sequence, one after the other, the state in registers.
// Everything here is 32-bit arithmetic; only the normed, gated output of delta_step is rounded.
#include "common.cuh"

namespace {

constexpr int DP_WARPS = 8;
constexpr int DP_MAX_D = 256;

__device__ __forceinline__ float silu32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_dt(float z) { return z > 20.f ? z : log1pf(expf(z)); }

struct DeltaPrep {
    const float* proj;         // [T, ld]: q (G d), k (G d), v (H dv) from column 0; b and a from columns b_at, a_at
    long long ld;
    int b_at, a_at;
    const float* taps_w;       // [taps, channels]
    float* state;              // per slot (taps - 1) * channels floats, oldest row first
    long long state_pitch;
    const float* a_log;        // [H]
    const float* dt_bias;      // [H]
    const int* seq_of_token;
    const int* cu_seqlens;
    const int* slots;
    int num_tokens, taps, H, G, d, dv, shift;
    float eps, q_scale;
    float* out;                // [T, channels]: q, k, v
    float* step;               // [T, 2 H]: beta, logarithm of the decay
};

// W neighbouring channels of row t convolved and passed through silu; `st`: the sequence's state, li: the row's place
// among the sequence's rows of the step.  With `shift` (one row a sequence) the state's rows move one place down.
template <int W, int TAPS>
__device__ __forceinline__ void conv_silu(const DeltaPrep& p, int t, int li, float* st, int ch, int channels, float* y) {
    const int taps = TAPS > 0 ? TAPS : p.taps;
#pragma unroll
    for (int e = 0; e < W; e++) y[e] = 0.f;
#pragma unroll
    for (int j = 0; j < taps; j++) {
        const int r = li - (taps - 1) + j;
        const float* src = r >= 0 ? p.proj + (size_t)(t - li + r) * p.ld + ch : st + (size_t)(taps - 1 + r) * channels + ch;
        const float* wj = p.taps_w + (size_t)j * channels + ch;
        if (W == 4) {
            const float4 x = *reinterpret_cast<const float4*>(src), w = *reinterpret_cast<const float4*>(wj);
            y[0] = fmaf(w.x, x.x, y[0]), y[1] = fmaf(w.y, x.y, y[1]), y[2] = fmaf(w.z, x.z, y[2]), y[3] = fmaf(w.w, x.w, y[3]);
            if (p.shift && j >= 1) *reinterpret_cast<float4*>(st + (size_t)(j - 1) * channels + ch) = x;
        } else {
            const float x = *src;
            y[0] = fmaf(*wj, x, y[0]);
            if (p.shift && j >= 1) st[(size_t)(j - 1) * channels + ch] = x;
        }
    }
#pragma unroll
    for (int e = 0; e < W; e++) y[e] = silu32(y[e]);
}

// grid (token, parts of its heads); a warp takes one head of q or k, or one run of 32 W channels of v, in turn.
template <int W, int TAPS>
__global__ void __launch_bounds__(DP_WARPS * 32)
delta_prepare_kernel(const DeltaPrep p) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x;
    const int qk = 2 * p.G * p.d, channels = qk + p.H * p.dv;
    const int vruns = (p.H * p.dv + 32 * W - 1) / (32 * W);
    const int items = 2 * p.G + vruns + 1;
    pdl_sync();
    const int s = p.seq_of_token[t];
    float* out = p.out + (size_t)t * channels;
    float* stp = p.step + (size_t)t * 2 * p.H;
    const int li = s >= 0 ? t - p.cu_seqlens[s] : 0;
    float* st = (s >= 0 && p.taps > 1) ? p.state + (size_t)p.slots[s] * p.state_pitch : nullptr;
    for (int item = blockIdx.y * DP_WARPS + warp; item < items; item += gridDim.y * DP_WARPS) {
        if (s < 0) {           // a row of no sequence: something finite, no state touched
            if (item < 2 * p.G) {
                for (int e = lane; e < p.d; e += 32) out[item * p.d + e] = 0.f;
            } else if (item < 2 * p.G + vruns) {
                for (int e = (item - 2 * p.G) * 32 * W + lane; e < min(p.H * p.dv, (item - 2 * p.G + 1) * 32 * W); e += 32)
                    out[qk + e] = 0.f;
            } else {
                for (int h = lane; h < 2 * p.H; h += 32) stp[h] = 0.f;
            }
            continue;
        }
        if (item < 2 * p.G) {
            const int ch0 = item * p.d;
            constexpr int PASSES = DP_MAX_D / (32 * W);
            float y[PASSES][W];
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < PASSES; i++) {
                const int e = (i * 32 + lane) * W;
                if (e < p.d) {
                    conv_silu<W, TAPS>(p, t, li, st, ch0 + e, channels, y[i]);
#pragma unroll
                    for (int z = 0; z < W; z++) ss = fmaf(y[i][z], y[i][z], ss);
                }
            }
            ss = warp_sum(ss);
            float inv = 1.0f / sqrtf(ss + p.eps);
            if (item < p.G) inv *= p.q_scale;
#pragma unroll
            for (int i = 0; i < PASSES; i++) {
                const int e = (i * 32 + lane) * W;
                if (e < p.d) {
                    if (W == 4)
                        *reinterpret_cast<float4*>(out + ch0 + e) =
                            make_float4(y[i][0] * inv, y[i][1 % W] * inv, y[i][2 % W] * inv, y[i][3 % W] * inv);
                    else
                        out[ch0 + e] = y[i][0] * inv;
                }
            }
        } else if (item < 2 * p.G + vruns) {
            const int e = ((item - 2 * p.G) * 32 + lane) * W;
            if (e < p.H * p.dv) {
                float y[W];
                conv_silu<W, TAPS>(p, t, li, st, qk + e, channels, y);
                if (W == 4)
                    *reinterpret_cast<float4*>(out + qk + e) = make_float4(y[0], y[1 % W], y[2 % W], y[3 % W]);
                else
                    out[qk + e] = y[0];
            }
        } else {
            const float* row = p.proj + (size_t)t * p.ld;
            for (int h = lane; h < p.H; h += 32) {
                stp[h] = 1.0f / (1.0f + expf(-row[p.b_at + h]));
                stp[p.H + h] = -expf(p.a_log[h]) * softplus_dt(row[p.a_at + h] + p.dt_bias[h]);
            }
        }
    }
}

struct DeltaSeq {
    const float* qkv;          // [T, channels] prepared q, k, v
    const float* step;         // [T, 2 H]
    float* state;              // per slot H * d * dv floats ([head][d][dv]) from the pointer given
    long long state_pitch;
    const int* cu_seqlens;
    const int* slots;
    int H, G, d, dv;
};

// ---- one token a sequence --------------------------------------------------------------------------
// A block a (head, sequence): thread (cg, kp) holds four neighbouring columns of every KP-th row of S.  The
// state is asked for before the wait for the predecessor: nothing since the step before has written it.
template <typename OT, int UNITS>
__global__ void __launch_bounds__(256)
delta_step_kernel(const DeltaSeq p, const float* __restrict__ gate, long long ldg, const float* __restrict__ norm_w,
                  float norm_eps, const int* __restrict__ seq_of_token, int num_tokens, OT* __restrict__ out) {
    extern __shared__ __align__(16) float ds_smem[];         // k [d] | q [d] | u [dv] | parts [KP][dv]
    __shared__ float red[32];
    const int h = blockIdx.x, s = blockIdx.y, d = p.d, dv = p.dv;
    const int CG = dv / 4, KP = blockDim.x / CG, cg = threadIdx.x % CG, kp = threadIdx.x / CG;
    const bool worker = kp < KP;
    float* sk = ds_smem;
    float* sq = sk + d;
    float* su = sq + d;
    float* parts = su + dv;
    const int t = p.cu_seqlens[s];
    const bool live = p.cu_seqlens[s + 1] > t && t < num_tokens && seq_of_token[t] >= 0;
    float* S = p.state + (size_t)p.slots[s] * p.state_pitch + (size_t)h * d * dv;
    float4 r[UNITS];
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        const int row = kp + i * KP;
        r[i] = (live && worker && row < d) ? *reinterpret_cast<const float4*>(S + (size_t)row * dv + cg * 4)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_sync();
    if (!live) {                                             // row s is a row of no sequence: something finite
        if (s < num_tokens && seq_of_token[s] < 0)
            for (int c = threadIdx.x; c < dv; c += blockDim.x) st_f(out + ((size_t)s * p.H + h) * dv + c, 0.f);
        return;
    }
    const int g = h / (p.H / p.G), channels = 2 * p.G * d + p.H * dv;
    const float* row = p.qkv + (size_t)t * channels;
    for (int i = threadIdx.x; i < d; i += blockDim.x) sq[i] = row[(size_t)g * d + i], sk[i] = row[(size_t)(p.G + g) * d + i];
    const float beta = p.step[(size_t)t * 2 * p.H + h], decay = expf(p.step[(size_t)t * 2 * p.H + p.H + h]);
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        const int rr = kp + i * KP;
        r[i].x *= decay, r[i].y *= decay, r[i].z *= decay, r[i].w *= decay;
        if (worker && rr < d) {
            const float k = sk[rr];
            acc.x = fmaf(k, r[i].x, acc.x), acc.y = fmaf(k, r[i].y, acc.y);
            acc.z = fmaf(k, r[i].z, acc.z), acc.w = fmaf(k, r[i].w, acc.w);
        }
    }
    if (worker) *reinterpret_cast<float4*>(parts + (size_t)kp * dv + cg * 4) = acc;
    __syncthreads();
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float held = 0.f;
        for (int q = 0; q < KP; q++) held += parts[(size_t)q * dv + c];
        su[c] = beta * (row[(size_t)2 * p.G * d + (size_t)h * dv + c] - held);
    }
    __syncthreads();
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (worker) {
        const float4 u = *reinterpret_cast<const float4*>(su + cg * 4);
#pragma unroll
        for (int i = 0; i < UNITS; i++) {
            const int rr = kp + i * KP;
            if (rr < d) {
                const float k = sk[rr], q = sq[rr];
                r[i].x = fmaf(k, u.x, r[i].x), r[i].y = fmaf(k, u.y, r[i].y), r[i].z = fmaf(k, u.z, r[i].z), r[i].w = fmaf(k, u.w, r[i].w);
                acc.x = fmaf(q, r[i].x, acc.x), acc.y = fmaf(q, r[i].y, acc.y);
                acc.z = fmaf(q, r[i].z, acc.z), acc.w = fmaf(q, r[i].w, acc.w);
                *reinterpret_cast<float4*>(S + (size_t)rr * dv + cg * 4) = r[i];
            }
        }
        *reinterpret_cast<float4*>(parts + (size_t)kp * dv + cg * 4) = acc;
    }
    __syncthreads();
    // the output's norm over the head and its gate
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float o = 0.f;
        for (int q = 0; q < KP; q++) o += parts[(size_t)q * dv + c];
        su[c] = o;
        ss = fmaf(o, o, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + norm_eps);
    for (int c = threadIdx.x; c < dv; c += blockDim.x)
        st_f(out + ((size_t)t * p.H + h) * dv + c,
             su[c] * inv * norm_w[(size_t)h * dv + c] * silu32(gate[(size_t)t * ldg + (size_t)h * dv + c]));
}

// ---- several tokens a sequence, one after the other ----------------------------------------------------
// grid (ceil(dv / 64), heads, sequences), KP * 16 threads: thread (kp = tid % KP, cg = tid / KP) holds rows
// kp * RPT ... of four neighbouring columns of S in registers (rows beyond d stay zero).  A run of TOK tokens is
// staged in shared memory as [k | q | the block's columns of v | beta | decay] a token, the next run's loads in
// flight while this one is worked on.  From one token to the next only S is carried, so the chain is: product
// with k, its sum over the KP threads, u, the update; the product with q hangs off it.
constexpr int DS_CPT = 4, DS_CG = 16, DS_COLS = DS_CPT * DS_CG;

template <int RPT, int KP, int TOK>
__global__ void __launch_bounds__(KP * DS_CG)
delta_scan_kernel(const DeltaSeq p, float* __restrict__ o) {
    constexpr int NP = RPT * KP, THREADS = KP * DS_CG;
    constexpr int PER_TOK = 2 * NP + DS_COLS + 2;
    constexpr int ROWLEN = (PER_TOK + 3) & ~3;
    constexpr int XPT = (PER_TOK + THREADS - 1) / THREADS;
    extern __shared__ __align__(16) float sm[];               // [TOK][ROWLEN]
    const int tid = threadIdx.x, kp = tid % KP, cg = tid / KP;
    const int h = blockIdx.y, s = blockIdx.z, g = h / (p.H / p.G), d = p.d, dv = p.dv;
    const int c0 = blockIdx.x * DS_COLS, col = c0 + cg * DS_CPT;
    pdl_sync();
    const int tok0 = p.cu_seqlens[s], cnt = p.cu_seqlens[s + 1] - tok0;
    if (cnt <= 0) return;
    const int channels = 2 * p.G * d + p.H * dv;
    float* S = p.state + (size_t)p.slots[s] * p.state_pitch + (size_t)h * d * dv;
    const bool vec = dv % 4 == 0 && ((uintptr_t)S) % 16 == 0;
    float sreg[RPT][DS_CPT];
#pragma unroll
    for (int m = 0; m < RPT; m++) {
        const int n = kp * RPT + m;
        if (vec && n < d && col < dv) {
            const float4 t4 = *reinterpret_cast<const float4*>(S + (size_t)n * dv + col);
            sreg[m][0] = t4.x, sreg[m][1] = t4.y, sreg[m][2] = t4.z, sreg[m][3] = t4.w;
        } else {
#pragma unroll
            for (int c = 0; c < DS_CPT; c++) sreg[m][c] = (n < d && col + c < dv) ? S[(size_t)n * dv + col + c] : 0.f;
        }
    }
    // what this thread brings into shared memory of every token; where each element comes from is worked out once
    const float* src[XPT];
    long long pitch[XPT];
#pragma unroll
    for (int e = 0; e < XPT; e++) {
        const int x = tid + e * THREADS;
        src[e] = nullptr, pitch[e] = channels;
        if (x < NP) {
            if (x < d) src[e] = p.qkv + (size_t)tok0 * channels + (size_t)(p.G + g) * d + x;
        } else if (x < 2 * NP) {
            if (x - NP < d) src[e] = p.qkv + (size_t)tok0 * channels + (size_t)g * d + (x - NP);
        } else if (x < 2 * NP + DS_COLS) {
            const int c = c0 + x - 2 * NP;
            if (c < dv) src[e] = p.qkv + (size_t)tok0 * channels + (size_t)2 * p.G * d + (size_t)h * dv + c;
        } else if (x < PER_TOK) {
            src[e] = p.step + (size_t)tok0 * 2 * p.H + (x - 2 * NP - DS_COLS) * p.H + h, pitch[e] = 2 * p.H;
        }
    }
    float ahead[TOK][XPT];
    auto fetch = [&](int t0) {
        const int nt = min(TOK, cnt - t0);
#pragma unroll
        for (int tt = 0; tt < TOK; tt++) {
            const long long r = t0 + min(tt, nt - 1);
#pragma unroll
            for (int e = 0; e < XPT; e++) ahead[tt][e] = src[e] ? src[e][r * pitch[e]] : 0.f;
        }
    };
    fetch(0);
    const bool b0 = (kp & 1) != 0, b1 = (kp & 2) != 0;
    // sums over the KP threads of a column group: afterwards every thread holds one column's, chosen by its
    // lowest two bits (each thread drops the columns another one carries on)
    auto reduce = [&](const float (&a)[2][DS_CPT]) {
        const float p0 = a[0][0] + a[1][0], p1 = a[0][1] + a[1][1], p2 = a[0][2] + a[1][2], p3 = a[0][3] + a[1][3];
        float v0 = (b0 ? p2 : p0) + __shfl_xor_sync(0xffffffffu, b0 ? p0 : p2, 1);
        const float v1 = (b0 ? p3 : p1) + __shfl_xor_sync(0xffffffffu, b0 ? p1 : p3, 1);
        v0 = (b1 ? v1 : v0) + __shfl_xor_sync(0xffffffffu, b1 ? v0 : v1, 2);
#pragma unroll
        for (int off = 4; off < KP; off <<= 1) v0 += __shfl_xor_sync(0xffffffffu, v0, off);
        return v0;
    };
    const int lane = tid & 31, group = lane & ~(KP - 1), my_col = (b0 ? 2 : 0) + (b1 ? 1 : 0);
    for (int t0 = 0; t0 < cnt; t0 += TOK) {
        const int nt = min(TOK, cnt - t0);
        __syncthreads();                     // the run before is no longer read
#pragma unroll
        for (int tt = 0; tt < TOK; tt++)
#pragma unroll
            for (int e = 0; e < XPT; e++) {
                const int x = tid + e * THREADS;
                if (x < PER_TOK) sm[tt * ROWLEN + x] = x == PER_TOK - 1 ? expf(ahead[tt][e]) : ahead[tt][e];
            }
        __syncthreads();
        if (t0 + TOK < cnt) fetch(t0 + TOK);
#pragma unroll 2
        for (int tt = 0; tt < nt; tt++) {
            const float* row = sm + tt * ROWLEN;
            const float beta = row[2 * NP + DS_COLS], decay = row[2 * NP + DS_COLS + 1];
            float kr[RPT];
            float acc[2][DS_CPT] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int m0 = 0; m0 < RPT; m0 += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(row + kp * RPT + m0);
                kr[m0] = k4.x, kr[m0 + 1] = k4.y, kr[m0 + 2] = k4.z, kr[m0 + 3] = k4.w;
#pragma unroll
                for (int z = 0; z < 4; z++)
#pragma unroll
                    for (int c = 0; c < DS_CPT; c++) {
                        sreg[m0 + z][c] *= decay;
                        acc[z & 1][c] = fmaf(kr[m0 + z], sreg[m0 + z][c], acc[z & 1][c]);
                    }
            }
            const float mine = beta * (row[2 * NP + cg * DS_CPT + my_col] - reduce(acc));
            // the column's u from the thread of the group that holds it: column c = 2 * bit0 + bit1 of its number
            float u[DS_CPT];
#pragma unroll
            for (int c = 0; c < DS_CPT; c++) u[c] = __shfl_sync(0xffffffffu, mine, group + ((c >> 1) | ((c & 1) << 1)));
            float oc[2][DS_CPT] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int m0 = 0; m0 < RPT; m0 += 4) {
                const float4 q4 = *reinterpret_cast<const float4*>(row + NP + kp * RPT + m0);
                const float qi[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                for (int z = 0; z < 4; z++)
#pragma unroll
                    for (int c = 0; c < DS_CPT; c++) {
                        sreg[m0 + z][c] = fmaf(kr[m0 + z], u[c], sreg[m0 + z][c]);
                        oc[z & 1][c] = fmaf(qi[z], sreg[m0 + z][c], oc[z & 1][c]);
                    }
            }
            const float ov = reduce(oc);
            if (kp < 4 && col + my_col < dv) o[(size_t)(tok0 + t0 + tt) * p.H * dv + (size_t)h * dv + col + my_col] = ov;
        }
    }
#pragma unroll
    for (int m = 0; m < RPT; m++) {
        const int n = kp * RPT + m;
        if (n >= d) continue;
        if (vec && col < dv) {
            *reinterpret_cast<float4*>(S + (size_t)n * dv + col) = make_float4(sreg[m][0], sreg[m][1], sreg[m][2], sreg[m][3]);
        } else {
#pragma unroll
            for (int c = 0; c < DS_CPT; c++)
                if (col + c < dv) S[(size_t)n * dv + col + c] = sreg[m][c];
        }
    }
}

bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace

// proj: [T, ld] 32-bit: q (G * d columns), k (G * d), v (H * dv), b and a (a column a value head) from b_at and
// a_at; taps_w: [taps, channels]; state: (taps - 1) * channels floats a slot from the pointer given; out: [T, channels]
// 32-bit; step: [T, 2 H] 32-bit (beta, then the decay's logarithm).  `shift`: the step brings one token a sequence and the state moves on here.
MOE_API int moe_delta_prepare(const float* proj, long long ld, int b_at, int a_at, const float* taps_w, int taps,
                              float* state, long long state_pitch, const float* a_log, const float* dt_bias,
                              const int* seq_of_token, const int* cu_seqlens, const int* slots, int num_tokens, int H,
                              int G, int d, int dv, float eps, float q_scale, int shift, float* out, float* step,
                              cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    const long long channels = 2LL * G * d + (long long)H * dv;
    if (!proj || !taps_w || !a_log || !dt_bias || !seq_of_token || !cu_seqlens || !slots || !out || !step || H <= 0 || G <= 0 ||
        H % G || d <= 0 || d > DP_MAX_D || dv <= 0 || taps < 1 || taps > 16 || (taps > 1 && !state) || ld < channels ||
        b_at < 0 || a_at < 0 || b_at + H > ld || a_at + H > ld || (taps > 1 && state_pitch < (taps - 1) * channels))
        return (int)cudaErrorInvalidValue;
    const DeltaPrep p{proj, ld, b_at, a_at, taps_w, state, state_pitch, a_log, dt_bias, seq_of_token, cu_seqlens, slots,
                      num_tokens, taps, H, G, d, dv, shift, eps, q_scale, out, step};
    const bool vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && state_pitch % 4 == 0 && aligned16(proj) && aligned16(taps_w) &&
                     aligned16(state) && aligned16(out);
    const int per = vec ? 128 : 32;
    const int items = 2 * G + (H * dv + per - 1) / per + 1;
    // few tokens: a warp an item; many: a block a token
    const dim3 grid(num_tokens, num_tokens >= 128 ? 1 : (items + DP_WARPS - 1) / DP_WARPS);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define PREP(W_, T_) return launch_pdl(delta_prepare_kernel<W_, T_>, grid, dim3(DP_WARPS * 32), 0, stream, p)
    if (vec) {
        if (taps == 2) PREP(4, 2);
        if (taps == 3) PREP(4, 3);
        if (taps == 4) PREP(4, 4);
        PREP(4, 0);
    }
    if (taps == 4) PREP(1, 4);
    PREP(1, 0);
#undef PREP
}

// One token a sequence.  qkv, step: as moe_delta_prepare leaves them; state: H * d * dv floats a slot from the pointer
// given; gate: [T, H * dv] 32-bit logits, rows of ldg; norm_w: [H * dv]; out: [T, H * dv] in out_dt (rows of no
// sequence become zeros).  Returns -1, with nothing launched, for sizes it does not take.
MOE_API int moe_delta_step(const float* qkv, const float* step, float* state, long long state_pitch, const float* gate,
                           long long ldg, const float* norm_w, float norm_eps, const int* seq_of_token,
                           const int* cu_seqlens, const int* slots, int num_tokens, int num_seqs, int H, int G, int d,
                           int dv, void* out, int out_dt, cudaStream_t stream) {
    if (num_seqs <= 0 || num_tokens <= 0) return 0;
    if (!qkv || !step || !state || !gate || !norm_w || !seq_of_token || !cu_seqlens || !slots || !out || H <= 0 || G <= 0 ||
        H % G || d <= 0 || dv <= 0 || ldg < (long long)H * dv || state_pitch < (long long)H * d * dv || num_seqs > 65535)
        return (int)cudaErrorInvalidValue;
    if (dv % 4 || dv > 512 || d > 256 || state_pitch % 4 || !aligned16(state)) return -1;
    const int cg = dv / 4, kp = 256 / cg, units = (d + kp - 1) / kp;
    const size_t smem = ((size_t)2 * ((d + 1) / 2 * 2) + dv + (size_t)kp * dv) * sizeof(float);
    if (units > 32 || smem > 48 * 1024 || d % 2) return -1;
    const DeltaSeq p{qkv, step, state, state_pitch, cu_seqlens, slots, H, G, d, dv};
#define STEP(OT_, U_)                                                                                                  \
    return launch_pdl(delta_step_kernel<OT_, U_>, dim3(H, num_seqs), dim3(256), smem, stream, p, gate, ldg, norm_w, norm_eps, \
                      seq_of_token, num_tokens, (OT_*)out)
#define STEP_U(OT_)                                                                                                    \
    do {                                                                                                               \
        if (units <= 4) STEP(OT_, 4);                                                                                  \
        if (units <= 8) STEP(OT_, 8);                                                                                  \
        if (units <= 16) STEP(OT_, 16);                                                                                \
        STEP(OT_, 32);                                                                                                 \
    } while (0)
    if (out_dt == DT_F32) STEP_U(float);
    STEP_U(__nv_bfloat16);
#undef STEP_U
#undef STEP
}

// Several tokens a sequence; o: [T, H * dv] 32-bit (rows of no sequence are left alone).
MOE_API int moe_delta_scan(const float* qkv, const float* step, float* state, long long state_pitch, const int* cu_seqlens,
                           const int* slots, int num_seqs, int H, int G, int d, int dv, float* o, cudaStream_t stream) {
    if (num_seqs <= 0) return 0;
    if (!qkv || !step || !state || !cu_seqlens || !slots || !o || H <= 0 || G <= 0 || H % G || d <= 0 || d > 256 || dv <= 0 ||
        state_pitch < (long long)H * d * dv || H > 65535 || num_seqs > 65535)
        return (int)cudaErrorInvalidValue;
    const DeltaSeq p{qkv, step, state, state_pitch, cu_seqlens, slots, H, G, d, dv};
    const dim3 grid((dv + DS_COLS - 1) / DS_COLS, H, num_seqs);
#define SCAN(RPT_, KP_, TOK_)                                                                                          \
    return launch_pdl(delta_scan_kernel<RPT_, KP_, TOK_>, grid, dim3(KP_ * DS_CG),                                     \
                      (size_t)(TOK_) * ((2 * RPT_ * KP_ + DS_COLS + 2 + 3) / 4 * 4) * sizeof(float), stream, p, o)
    if (d <= 32) SCAN(4, 8, 16);
    if (d <= 64) SCAN(8, 8, 16);
    if (d <= 128) SCAN(16, 8, 16);
    SCAN(16, 16, 16);
#undef SCAN
}
