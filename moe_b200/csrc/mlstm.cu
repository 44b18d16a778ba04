// An exponentially gated matrix memory (mLSTM): a recurrent mixer whose state is written with a gate exp(i) and kept
// with a gate f in (0, 1), both one number a head and token, in units of exp(m) for a running maximum m.
//
// Per head, with log gates lf = logsigmoid(cap tanh(f_raw / cap)), li = cap tanh(i_raw / cap) (their biases added first)
// and S [d, dv], n [d] and m that start at zero:
//   m' = max(lf + m, li);  a = e^(lf + m - m');  b = e^(li - m');  m <- m'
//   S <- a S + b k v^T;  n <- a n + b k;  o = S^T q / (max(|n . q|, e^(-m)) + 1e-6)
//
//   mlstm_gates   a, b and e^(-m) of every token, and the sequences' m moved on: a block a (head, sequence), a token a
//                 thread (the pairs (lf, li) compose as m -> max(lf + m, li), an associative operation).
//   mlstm_scan    several tokens a sequence, four at a time, state and normaliser in registers.
//   mlstm_step    one token a sequence: gates, recurrence with the state read once and written once, and the output's
//                 norm and gate behind it, a block a (head, sequence).
// Everything is 32-bit arithmetic; only the normed, gated output of mlstm_step is rounded.
#include "common.cuh"

namespace {

constexpr float READ_EPS = 1e-6f;

__device__ __forceinline__ float log_in(float raw, float cap) { return cap * tanhf(raw / cap); }
__device__ __forceinline__ float log_keep(float raw, float cap) { return log_sigmoid(cap * tanhf(raw / cap)); }

struct MemSeq {
    const float* proj;         // [T, ld] 32-bit: q (H d) from q_at, k (H d) from k_at, v (H dv) from v_at, i and f logits (H each)
    long long ld;
    int q_at, k_at, v_at, i_at, f_at;
    const float* i_bias;       // [H]
    const float* f_bias;       // [H]
    float* state;              // per slot S [H][d][dv] | n [copies][H][d] | m [H] from the pointer given
    long long state_pitch;
    const int* cu_seqlens;
    const int* slots;
    float* steps;              // [T, 3 H]: a, b, e^(-m)
    int H, d, dv;
    float cap, q_scale;
    int copies;                // of n, one for every 16 columns of S: blocks that share a head have ones of their own
    __device__ __forceinline__ size_t n_at(int copy, int h) const { return (size_t)H * d * dv + ((size_t)copy * H + h) * d; }
    __device__ __forceinline__ size_t m_at(int h) const { return (size_t)H * d * (dv + copies) + h; }
};

// grid (H, sequences); any whole number of warps: a chunk of as many tokens as threads at a time
__global__ void __launch_bounds__(1024)
mlstm_gates_kernel(const MemSeq p) {
    __shared__ float wf[32], wi[32];                  // a warp's tokens as one pair
    pdl_sync();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5, h = blockIdx.x, s = blockIdx.y;
    const int tok0 = p.cu_seqlens[s], cnt = p.cu_seqlens[s + 1] - tok0;
    if (cnt <= 0) return;
    float* m_at = p.state + (size_t)p.slots[s] * p.state_pitch + p.m_at(h);
    const float ib = p.i_bias[h], fb = p.f_bias[h];
    float m = *m_at;
    for (int t0 = 0; t0 < cnt; t0 += blockDim.x) {
        const int t = t0 + threadIdx.x;
        const bool on = t < cnt;                      // (places beyond the last token leave m as it is)
        const float* row = p.proj + (size_t)(tok0 + min(t, cnt - 1)) * p.ld;
        const float li = on ? log_in(row[p.i_at + h] + ib, p.cap) : -INFINITY;
        const float lf = on ? log_keep(row[p.f_at + h] + fb, p.cap) : 0.f;
        float cf = lf, ci = li;                       // the warp's tokens up to this one as one pair
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, cf, o), pi = __shfl_up_sync(0xffffffffu, ci, o);
            if (lane >= o) ci = fmaxf(cf + pi, ci), cf += pf;
        }
        if (lane == 31) wf[warp] = cf, wi[warp] = ci;
        __syncthreads();
        float before = m, mine = m;                   // m in front of the warp, and at the end of the chunk
        for (int w = 0; w < warps; w++) {
            if (w == warp) mine = before;
            before = fmaxf(wf[w] + before, wi[w]);
        }
        m = before;
        const float after = fmaxf(cf + mine, ci);
        before = __shfl_up_sync(0xffffffffu, after, 1);
        if (lane == 0) before = mine;
        if (on) {
            float* out = p.steps + (size_t)(tok0 + t) * 3 * p.H + h;
            out[0] = expf(fminf(lf + before - after, 0.f));
            out[p.H] = expf(fminf(li - after, 0.f));
            out[2 * p.H] = expf(-after);
        }
        __syncthreads();                              // the pairs are read before the next chunk's are written
    }
    if (threadIdx.x == 0) *m_at = m;
}

// ---- one token a sequence --------------------------------------------------------------------------
// A block a (head, sequence): thread (cg, kp) holds four neighbouring columns of every KP-th row of S, asked for before
// the wait for the predecessor (nothing since the step before has written it).
template <typename OT, int UNITS>
__global__ void __launch_bounds__(256)
mlstm_step_kernel(const MemSeq p, const float* __restrict__ gate, long long ldg, const float* __restrict__ norm_w,
                  float norm_eps, const int* __restrict__ seq_of_token, int num_tokens, int gate_fn, OT* __restrict__ out) {
    extern __shared__ __align__(16) float ms_smem[];         // k [d] | q [d] | o [dv] | parts [KP][dv]
    __shared__ float red[32];
    const int h = blockIdx.x, s = blockIdx.y, d = p.d, dv = p.dv;
    const int CG = dv / 4, KP = blockDim.x / CG, cg = threadIdx.x % CG, kp = threadIdx.x / CG;
    const bool worker = kp < KP;
    const int dp = (d + 3) & ~3;
    float* sk = ms_smem;
    float* sq = sk + dp;
    float* so = sq + dp;
    float* parts = so + dv;
    const int t = p.cu_seqlens[s];
    const bool live = p.cu_seqlens[s + 1] > t && t < num_tokens && seq_of_token[t] >= 0;
    float* base = p.state + (size_t)p.slots[s] * p.state_pitch;
    float* S = base + (size_t)h * d * dv;
    float* N = base + p.n_at(0, h);
    float* m_at = base + p.m_at(h);
    float4 r[UNITS];
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        const int row = kp + i * KP;
        r[i] = (live && worker && row < d) ? *reinterpret_cast<const float4*>(S + (size_t)row * dv + cg * 4)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float held = (live && (int)threadIdx.x < d) ? N[threadIdx.x] : 0.f;      // (d <= 256)
    const float m0 = live ? *m_at : 0.f;
    pdl_sync();
    if (!live) {                                             // row s is a row of no sequence: something finite
        if (s < num_tokens && seq_of_token[s] < 0)
            for (int c = threadIdx.x; c < dv; c += blockDim.x) st_f(out + ((size_t)s * p.H + h) * dv + c, 0.f);
        return;
    }
    const float* row = p.proj + (size_t)t * p.ld;
    const float li = log_in(row[p.i_at + h] + p.i_bias[h], p.cap), lf = log_keep(row[p.f_at + h] + p.f_bias[h], p.cap);
    const float m1 = fmaxf(lf + m0, li), a = expf(lf + m0 - m1), b = expf(li - m1);
    float nq = 0.f;
    if ((int)threadIdx.x < d) {
        const int i = threadIdx.x;
        const float k = row[p.k_at + h * d + i], q = row[p.q_at + h * d + i] * p.q_scale, n = fmaf(a, held, b * k);
        sk[i] = b * k, sq[i] = q;
        for (int c = 0; c < p.copies; c++) N[(size_t)c * p.H * d + i] = n;
        nq = n * q;
    }
    nq = block_sum(nq, red);                                 // (its barrier also shows sk and sq to everyone)
    const float inv_read = 1.0f / (fmaxf(fabsf(nq), expf(-m1)) + READ_EPS);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (worker) {
        const float* v = row + p.v_at + (size_t)h * dv + cg * 4;
        const float v0 = v[0], v1 = v[1], v2 = v[2], v3 = v[3];
#pragma unroll
        for (int i = 0; i < UNITS; i++) {
            const int rr = kp + i * KP;
            if (rr < d) {
                const float k = sk[rr], q = sq[rr];
                r[i].x = fmaf(a, r[i].x, k * v0), r[i].y = fmaf(a, r[i].y, k * v1);
                r[i].z = fmaf(a, r[i].z, k * v2), r[i].w = fmaf(a, r[i].w, k * v3);
                acc.x = fmaf(q, r[i].x, acc.x), acc.y = fmaf(q, r[i].y, acc.y);
                acc.z = fmaf(q, r[i].z, acc.z), acc.w = fmaf(q, r[i].w, acc.w);
                *reinterpret_cast<float4*>(S + (size_t)rr * dv + cg * 4) = r[i];
            }
        }
        *reinterpret_cast<float4*>(parts + (size_t)kp * dv + cg * 4) = acc;
    }
    if (threadIdx.x == 0) *m_at = m1;
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float o = 0.f;
        for (int q = 0; q < KP; q++) o += parts[(size_t)q * dv + c];
        o *= inv_read;
        so[c] = o;
        ss = fmaf(o, o, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + norm_eps);
    for (int c = threadIdx.x; c < dv; c += blockDim.x)
        st_f(out + ((size_t)t * p.H + h) * dv + c,
             so[c] * inv * norm_w[(size_t)h * dv + c] * gate_value(gate_fn, gate[(size_t)t * ldg + (size_t)h * dv + c]));
}

// ---- several tokens a sequence: four at a time ------------------------------------------------------------
// With A_i the product of a from a group's first token to its i-th, P_ij that from the one after j to i, and S, n the
// state before the group,
//     S^T q_i -> A_i S^T q_i + sum_(j<=i) P_ij b_j (q_i . k_j) v_j,   n . q_i -> A_i n . q_i + sum_(j<=i) P_ij b_j (q_i . k_j)
//     S <- A_4 S + sum_j P_4j b_j k_j v_j^T,                          n <- A_4 n + sum_j P_4j b_j k_j
// which is the recurrence written out.  The normaliser n is one more column of S whose value is always 1.
//
// grid (ceil(dv / COLS), heads, sequences), 128 threads: thread (kp = tid % KP, cg = tid / KP) holds four neighbouring
// columns of rows 4 kp ... 4 kp + 3 of every 4 KP rows of S in registers, and the same rows of n (every column group
// for itself).  KP = 16 (32 columns a block) or, where those blocks would leave SMs idle, 32 (16 columns a block, half as
// many rows a thread).  A run of sixteen tokens is staged in shared memory as [k | q | the block's columns of v] a token
// (cp.async, two buffers; places beyond the sequence's last token are zeros with a = 1, b = 0); warp w forms the
// scalars of the run's group w.  Within a run the groups follow one another without a block barrier.
constexpr int MG = 4, MRUN = 16, MTHREADS = 128, COPY_COLS = 16;
__host__ __device__ constexpr int mcols(int kp) { return 4 * (MTHREADS / kp); }
constexpr int MCOEF = 36;      // a group's scalars: [0, 16) c_ij of token i in row i, [16, 20) A_i, [20, 24) P_4j b_j, [24, 28) e^(-m_i)

__device__ __forceinline__ void cp_zfill(float* dst, const float* src, int bytes, bool on) {
    const unsigned at = (unsigned)__cvta_generic_to_shared(dst);
    const int n = on ? bytes : 0;
    if (bytes == 16)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(at), "l"(src), "r"(n) : "memory");
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(at), "l"(src), "r"(n) : "memory");
}

template <int RPT, int KP>
__host__ __device__ constexpr size_t mlstm_scan_floats() {
    return (size_t)2 * MRUN * (2 * RPT * KP + mcols(KP)) + 2 * 3 * MRUN + 4 * MCOEF;
}

// VEC: rows of q, k and v start on 16-byte boundaries and hold whole 16-byte units.
// Few, long sequences leave SMs idle and the chain over the tokens long: a sequence's tokens may be cut into segments
// that run side by side (a is one number a head and token, so a segment's effect on what follows is its own end from a
// zero start and the product of its a):
//   phase 1  every segment but a sequence's last: its end and that product into a workspace, no outputs; the first one
//            also copies the sequence's state there
//   phase 2  every segment: its start from that copy and the ends before it, then the recurrence with outputs; the last
//            segment that holds tokens writes the state back
// which changes the order of additions, nothing else.
struct MemSegments {
    int segs, seg_len;       // segments a sequence (1: none of this), tokens a segment (a multiple of the staged run)
    float* ends;             // [sequence][segs] planes of `pitch` floats, S then n as in the state; the last one: the copy
    long long pitch;
    float* products;         // [sequence][segs][H]
};

// PHASE (0: the whole sequence in one go; 1, 2: see above) is known when compiled.
template <int RPT, int KP, bool VEC, int PHASE>
__global__ void __launch_bounds__(MTHREADS, RPT == 4 ? 4 : RPT == 8 ? 3 : 1)
mlstm_scan_kernel(const MemSeq p, float* __restrict__ o, const MemSegments sg) {
    constexpr int NP = RPT * KP, MCOLS = mcols(KP);
    constexpr int ROWLEN = 2 * NP + MCOLS;
    extern __shared__ __align__(16) float sm[];               // [2][MRUN][ROWLEN] | scalars [4][MCOEF] | steps [2][3][MRUN]
    float* s_coef = sm + 2 * MRUN * ROWLEN;
    float* s_step = s_coef + 4 * MCOEF;
    const int tid = threadIdx.x, kp = tid % KP, cg = tid / KP, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, s = PHASE ? blockIdx.z / sg.segs : blockIdx.z, seg = PHASE ? blockIdx.z % sg.segs : 0, d = p.d, dv = p.dv;
    const int c0 = blockIdx.x * MCOLS, col = c0 + cg * 4;
    for (int i = tid; i < 2 * MRUN * ROWLEN; i += MTHREADS) sm[i] = 0.f;         // columns that no copy writes stay zero
    const int seq_cnt = p.cu_seqlens[s + 1] - p.cu_seqlens[s];
    const int tok0 = p.cu_seqlens[s] + (PHASE ? seg * sg.seg_len : 0);
    const int cnt = PHASE ? min(sg.seg_len, seq_cnt - seg * sg.seg_len) : seq_cnt;
    if (cnt <= 0) return;
    const bool last_seg = !PHASE || (seg + 1) * sg.seg_len >= seq_cnt;            // the last one that holds tokens
    if (PHASE == 1 && last_seg && seg > 0) return;                              // nothing comes after it
    const int ncols = min(MCOLS, dv - c0);
    const size_t s_off = (size_t)h * d * dv, n_off = p.n_at(blockIdx.x * (MCOLS / COPY_COLS), h);
    float* state = p.state + (size_t)p.slots[s] * p.state_pitch;
    float* planes = PHASE ? sg.ends + (size_t)s * sg.segs * sg.pitch : nullptr;
    const bool vec_state = dv % 4 == 0 && ((uintptr_t)(state + s_off)) % 16 == 0;
    float sreg[RPT][4], nreg[RPT];
    // this thread's part of S and n from the plane `from`, times `keep` what it holds plus it
    auto load = [&](const float* from, float keep) {
#pragma unroll
        for (int m = 0; m < RPT; m++) {
            const int n = (m / 4) * 4 * KP + kp * 4 + m % 4;
            if (n >= d) continue;
            nreg[m] = fmaf(keep, nreg[m], from[n_off + n]);
            const float* row = from + s_off + (size_t)n * dv + col;
            if (vec_state && col < dv) {
                const float4 t4 = *reinterpret_cast<const float4*>(row);
                sreg[m][0] = fmaf(keep, sreg[m][0], t4.x), sreg[m][1] = fmaf(keep, sreg[m][1], t4.y);
                sreg[m][2] = fmaf(keep, sreg[m][2], t4.z), sreg[m][3] = fmaf(keep, sreg[m][3], t4.w);
            } else {
#pragma unroll
                for (int c = 0; c < 4; c++)
                    if (col + c < dv) sreg[m][c] = fmaf(keep, sreg[m][c], row[c]);
            }
        }
    };
    auto store = [&](float* to) {
#pragma unroll
        for (int m = 0; m < RPT; m++) {
            const int n = (m / 4) * 4 * KP + kp * 4 + m % 4;
            if (n >= d) continue;
            float* row = to + s_off + (size_t)n * dv + col;
            if (vec_state && col < dv) {
                *reinterpret_cast<float4*>(row) = make_float4(sreg[m][0], sreg[m][1], sreg[m][2], sreg[m][3]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; c++)
                    if (col + c < dv) row[c] = sreg[m][c];
            }
            if (cg < MCOLS / COPY_COLS && blockIdx.x * (MCOLS / COPY_COLS) + cg < p.copies) to[n_off + (size_t)cg * p.H * d + n] = nreg[m];
        }
    };
    auto clear = [&]() {
#pragma unroll
        for (int m = 0; m < RPT; m++) nreg[m] = sreg[m][0] = sreg[m][1] = sreg[m][2] = sreg[m][3] = 0.f;
    };
    clear();
    if (PHASE == 0) load(state, 0.f);
    if (PHASE == 1 && seg == 0) {
        load(state, 0.f);
        store(planes + (size_t)(sg.segs - 1) * sg.pitch);
        if (last_seg) return;
        clear();
    }
    if (PHASE == 2) {
        load(planes + (size_t)(sg.segs - 1) * sg.pitch, 0.f);
        for (int q = 0; q < seg; q++) load(planes + (size_t)q * sg.pitch, sg.products[((size_t)s * sg.segs + q) * p.H + h]);
    }
    float product = 1.f;
    const float* base = p.proj + (size_t)tok0 * p.ld;
    const float* sbase = p.steps + (size_t)tok0 * 3 * p.H + h;
    const int k_at = p.k_at + h * d, q_at = p.q_at + h * d, v_at = p.v_at + h * dv + c0;
    auto stage = [&](int t0, int buf) {
        float* dst = sm + buf * MRUN * ROWLEN;
        constexpr int W = VEC ? 4 : 1;
        const int kw = d / W, vw = ncols / W, per = 2 * kw + vw;
        for (int tt = warp; tt < MRUN; tt += MTHREADS / 32) {           // a warp a token
            const bool on = t0 + tt < cnt;
            const float* row = base + (size_t)min(t0 + tt, cnt - 1) * p.ld;
            float* to = dst + tt * ROWLEN;
            for (int e = lane; e < per; e += 32) {
                const int x = e < kw ? e : e < 2 * kw ? e - kw : e - 2 * kw;
                cp_zfill(to + (e < kw ? 0 : e < 2 * kw ? NP : 2 * NP) + x * W, row + (e < kw ? k_at : e < 2 * kw ? q_at : v_at) + x * W, 4 * W, on);
            }
        }
        if (tid < 3 * MRUN) {
            const int tt = tid % MRUN, which = tid / MRUN;
            cp_zfill(s_step + (buf * 3 + which) * MRUN + tt, sbase + (size_t)min(t0 + tt, cnt - 1) * 3 * p.H + which * p.H, 4, t0 + tt < cnt);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    __syncthreads();                                  // the zeros are there before any copy writes
    stage(0, 0);
    const bool b0 = (kp & 1) != 0, b1 = (kp & 2) != 0, b2 = (kp & 4) != 0, b3 = (kp & 8) != 0;
    const int my_col = (b0 ? 2 : 0) + (b1 ? 1 : 0), my_tok = (b2 ? 2 : 0) + (b3 ? 1 : 0);
    for (int t0 = 0, buf = 0; t0 < cnt; t0 += MRUN, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                              // this run is there, and the one before is no longer read
        if (t0 + MRUN < cnt) stage(t0 + MRUN, buf ^ 1);
        const float* run = sm + buf * MRUN * ROWLEN;
        {
            // the scalars of group `warp`: products of its queries and keys, then everything made of them
            const float* row = run + warp * MG * ROWLEN;
            float dots[16];                           // q_i . k_j in place 4 i + j (j <= i)
#pragma unroll
            for (int i = 0; i < 16; i++) dots[i] = 0.f;
            for (int e = lane * 4; e < NP; e += 128) {
                float4 k4[MG], q4[MG];
#pragma unroll
                for (int i = 0; i < MG; i++) {
                    k4[i] = *reinterpret_cast<const float4*>(row + i * ROWLEN + e);
                    q4[i] = *reinterpret_cast<const float4*>(row + i * ROWLEN + NP + e);
                }
#pragma unroll
                for (int i = 0; i < MG; i++)
#pragma unroll
                    for (int j = 0; j <= i; j++)
                        dots[4 * i + j] = fmaf(q4[i].x, k4[j].x, fmaf(q4[i].y, k4[j].y, fmaf(q4[i].z, k4[j].z, fmaf(q4[i].w, k4[j].w, dots[4 * i + j]))));
            }
            // sixteen sums over the warp; lane l ends with number l & 15
            float v8[8], v4[4], v2[2];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const bool up = (lane & 8) != 0;
                v8[i] = (up ? dots[8 + i] : dots[i]) + __shfl_xor_sync(0xffffffffu, up ? dots[i] : dots[8 + i], 8);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const bool up = (lane & 4) != 0;
                v4[i] = (up ? v8[4 + i] : v8[i]) + __shfl_xor_sync(0xffffffffu, up ? v8[i] : v8[4 + i], 4);
            }
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const bool up = (lane & 2) != 0;
                v2[i] = (up ? v4[2 + i] : v4[i]) + __shfl_xor_sync(0xffffffffu, up ? v4[i] : v4[2 + i], 2);
            }
            const bool up = (lane & 1) != 0;
            float dot = (up ? v2[1] : v2[0]) + __shfl_xor_sync(0xffffffffu, up ? v2[0] : v2[1], 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 16);
            const float* sa = s_step + buf * 3 * MRUN + warp * MG;
            const float* sb = sa + MRUN;
            const float* se = sb + MRUN;
            const int left = cnt - t0 - warp * MG;    // tokens of the group; places beyond change nothing
            auto keep = [&](int i) { return i < left ? sa[i] : 1.f; };
            const int n = lane & 15, i = n >> 2, j = n & 3;
            if (lane < 16) {
                float c = j <= i ? dot * sb[j] * p.q_scale : 0.f;
                for (int e = j + 1; e <= i; e++) c *= keep(e);
                s_coef[warp * MCOEF + n] = c;
            } else if (n < 4) {
                float c = p.q_scale;
                for (int e = 0; e <= n; e++) c *= keep(e);
                s_coef[warp * MCOEF + 16 + n] = c;
            } else if (n < 8) {
                float c = sb[n - 4];
                for (int e = n - 3; e < MG; e++) c *= keep(e);
                s_coef[warp * MCOEF + 16 + n] = c;
            } else if (n < 12) {
                s_coef[warp * MCOEF + 16 + n] = se[n - 8];
            } else if (n == 12) {
                s_coef[warp * MCOEF + 28] = keep(0) * keep(1) * keep(2) * keep(3);
            }
        }
        __syncthreads();
        const int groups = (min(MRUN, cnt - t0) + MG - 1) / MG;
        for (int gr = 0; gr < groups; gr++) {
            const float* row = run + gr * MG * ROWLEN + kp * 4;
            const float* cf = s_coef + gr * MCOEF;
            const float* vgr = run + gr * MG * ROWLEN + 2 * NP + cg * 4;
            float hq[MG][4], hn[MG];
            if (PHASE == 1) product *= cf[28];
#pragma unroll
            for (int i = 0; i < MG; i++) {
                hn[i] = 0.f;
#pragma unroll
                for (int c = 0; c < 4; c++) hq[i][c] = 0.f;
            }
            float vb[MG][4];                          // P_4j b_j v_j
            float wb[MG];
            const float a4 = cf[28];
#pragma unroll
            for (int j = 0; j < MG; j++) {
                const float4 v4 = *reinterpret_cast<const float4*>(vgr + j * ROWLEN);
                wb[j] = cf[20 + j];
                vb[j][0] = wb[j] * v4.x, vb[j][1] = wb[j] * v4.y, vb[j][2] = wb[j] * v4.z, vb[j][3] = wb[j] * v4.w;
            }
#pragma unroll
            for (int m0 = 0; m0 < RPT; m0 += 4) {
#pragma unroll
                for (int i = 0; i < (PHASE == 1 ? 0 : MG); i++) {
                    const float4 q4 = *reinterpret_cast<const float4*>(row + i * ROWLEN + NP + m0 * KP);
                    const float qi[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int z = 0; z < 4; z++) {
                        hn[i] = fmaf(qi[z], nreg[m0 + z], hn[i]);
#pragma unroll
                        for (int c = 0; c < 4; c++) hq[i][c] = fmaf(qi[z], sreg[m0 + z][c], hq[i][c]);
                    }
                }
#pragma unroll
                for (int z = 0; z < 4; z++) {
                    nreg[m0 + z] *= a4;
#pragma unroll
                    for (int c = 0; c < 4; c++) sreg[m0 + z][c] *= a4;
                }
#pragma unroll
                for (int j = 0; j < MG; j++) {
                    const float4 k4 = *reinterpret_cast<const float4*>(row + j * ROWLEN + m0 * KP);
                    const float kj[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                    for (int z = 0; z < 4; z++) {
                        nreg[m0 + z] = fmaf(kj[z], wb[j], nreg[m0 + z]);
#pragma unroll
                        for (int c = 0; c < 4; c++) sreg[m0 + z][c] = fmaf(kj[z], vb[j][c], sreg[m0 + z][c]);
                    }
                }
            }
            if constexpr (PHASE != 1) {               // (phase 1: the end alone)
                // Sums over the threads of a column group; on the way every thread drops what another one carries
                // on: bits 0 and 1 of kp pick the column, bits 2 and 3 the token.
                float r2[MG][2], r1[MG], t2[2], n2[2];
#pragma unroll
                for (int i = 0; i < MG; i++)
#pragma unroll
                    for (int c = 0; c < 2; c++)
                        r2[i][c] = (b0 ? hq[i][2 + c] : hq[i][c]) + __shfl_xor_sync(0xffffffffu, b0 ? hq[i][c] : hq[i][2 + c], 1);
#pragma unroll
                for (int i = 0; i < MG; i++)
                    r1[i] = (b1 ? r2[i][1] : r2[i][0]) + __shfl_xor_sync(0xffffffffu, b1 ? r2[i][0] : r2[i][1], 2);
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    t2[i] = (b2 ? r1[2 + i] : r1[i]) + __shfl_xor_sync(0xffffffffu, b2 ? r1[i] : r1[2 + i], 4);
                    n2[i] = (b2 ? hn[2 + i] : hn[i]) + __shfl_xor_sync(0xffffffffu, b2 ? hn[i] : hn[2 + i], 4);
                }
                float read = (b3 ? t2[1] : t2[0]) + __shfl_xor_sync(0xffffffffu, b3 ? t2[0] : t2[1], 8);
                float size = (b3 ? n2[1] : n2[0]) + __shfl_xor_sync(0xffffffffu, b3 ? n2[0] : n2[1], 8);
                if (KP == 32) read += __shfl_xor_sync(0xffffffffu, read, 16), size += __shfl_xor_sync(0xffffffffu, size, 16);
                size += __shfl_xor_sync(0xffffffffu, size, 1);
                size += __shfl_xor_sync(0xffffffffu, size, 2);
                const float4 c4 = *reinterpret_cast<const float4*>(cf + 4 * my_tok);
                const float ai = cf[16 + my_tok];
                read = ai * read + c4.x * vgr[my_col] + c4.y * vgr[ROWLEN + my_col] + c4.z * vgr[2 * ROWLEN + my_col] + c4.w * vgr[3 * ROWLEN + my_col];
                size = ai * size + c4.x + c4.y + c4.z + c4.w;
                const int t = t0 + gr * MG + my_tok;
                if (kp < 16 && t < cnt && col + my_col < dv)
                    o[(size_t)(tok0 + t) * p.H * dv + (size_t)h * dv + col + my_col] = read / (fmaxf(fabsf(size), cf[24 + my_tok]) + READ_EPS);
            }
        }
    }
    if (PHASE == 1) {
        store(planes + (size_t)seg * sg.pitch);
        if (tid == 0 && blockIdx.x == 0) sg.products[((size_t)s * sg.segs + seg) * p.H + h] = product;
    } else if (last_seg) {
        store(state);
    }
}

bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace

// How a slot's state is laid out, in floats: S [heads][d][dv] | n [copies][heads][d] | m [heads]; the size in all.
MOE_API long long moe_mlstm_state_floats(int H, int d, int dv) {
    return (long long)H * d * (dv + (dv + COPY_COLS - 1) / COPY_COLS) + H;
}

static int mlstm_bad(const float* proj, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at, const float* i_bias,
                     const float* f_bias, const float* state, long long state_pitch, const int* cu_seqlens, const int* slots,
                     int H, int d, int dv, float cap) {
    if (!proj || !i_bias || !f_bias || !state || !cu_seqlens || !slots || H <= 0 || d <= 0 || d > 256 || dv <= 0 || !(cap > 0.f) ||
        q_at < 0 || k_at < 0 || v_at < 0 || i_at < 0 || f_at < 0 || q_at + H * d > ld || k_at + H * d > ld || v_at + H * dv > ld ||
        i_at + H > ld || f_at + H > ld || state_pitch < moe_mlstm_state_floats(H, d, dv) || H > 65535)
        return 1;
    return 0;
}

// proj: [T, ld] 32-bit with the columns of q (H * d), k (H * d), v (H * dv) and the gates' logits (H each) from the places
// given; i_bias, f_bias: [H]; state: moe_mlstm_state_floats floats a slot from the pointer given; longest: the most tokens a
// sequence brings (0: unknown); segs, seg_len, ends, pitch, products: MemSegments; steps: [T, 3 H] scratch, filled here; o: [T, H * dv] 32-bit (rows of no sequence are left alone).
MOE_API int moe_mlstm_scan(const float* proj, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                           const float* i_bias, const float* f_bias, float cap, float q_scale, float* state,
                           long long state_pitch, const int* cu_seqlens, const int* slots, int num_seqs, int H, int d,
                           int dv, float* steps, float* o, int longest, int segs,
                           int seg_len, float* ends, long long pitch, float* products, cudaStream_t stream) {
    if (num_seqs <= 0) return 0;
    if (!steps || !o || num_seqs > 65535 ||
        mlstm_bad(proj, ld, q_at, k_at, v_at, i_at, f_at, i_bias, f_bias, state, state_pitch, cu_seqlens, slots, H, d, dv, cap))
        return (int)cudaErrorInvalidValue;
    if (segs < 1 || (segs > 1 && (!ends || !products || seg_len <= 0 || seg_len % MRUN || pitch < moe_mlstm_state_floats(H, d, dv) - H ||
                                  pitch % 4 || (long long)num_seqs * segs > 65535)))
        return (int)cudaErrorInvalidValue;
    const int copies = (dv + COPY_COLS - 1) / COPY_COLS;
    const MemSeq p{proj, ld, q_at, k_at, v_at, i_at, f_at, i_bias, f_bias, state, state_pitch, cu_seqlens, slots, steps,
                   H, d, dv, cap, q_scale, copies};
    const int threads = longest > 0 && longest < 1024 ? (longest + 31) / 32 * 32 : 1024;
    int code = launch_pdl(mlstm_gates_kernel, dim3(H, num_seqs), dim3(threads), 0, stream, p);
    if (code) return code;
    // few blocks: the narrow form puts twice as many on the SMs
    const bool narrow = d > 64 && (long long)((dv + mcols(16) - 1) / mcols(16)) * H * num_seqs * segs * 2 <= scan_sms();
    const int cols = mcols(narrow ? 32 : 16);
    const dim3 grid((dv + cols - 1) / cols, H, num_seqs * segs);
    const MemSegments sg{segs, seg_len, ends, pitch, products};
    const bool vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && q_at % 4 == 0 && k_at % 4 == 0 && v_at % 4 == 0 && aligned16(proj);
    // (an ordinary launch: blocks placed while the kernel before still holds some SMs would be several to an SM beside
    // empty ones, and a scan is as slow as its most crowded SM)
#define SCAN_P(RPT_, KP_, V_, PH_)                                                                                     \
    do {                                                                                                               \
        const size_t smem = scan_smem(mlstm_scan_floats<RPT_, KP_>() * sizeof(float), (long long)grid.x * grid.y * grid.z); \
        if (smem > 48 * 1024) {                                                                                        \
            cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<RPT_, KP_, V_, PH_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                       \
        }                                                                                                              \
        mlstm_scan_kernel<RPT_, KP_, V_, PH_><<<grid, MTHREADS, smem, stream>>>(p, o, sg);                             \
        if (PH_ != 1) return launch_status();                                                                          \
    } while (0)
#define SCAN_V(RPT_, KP_, V_)                                                                                          \
    do {                                                                                                               \
        if (segs > 1) {                                                                                                \
            SCAN_P(RPT_, KP_, V_, 1);                                                                                  \
            SCAN_P(RPT_, KP_, V_, 2);                                                                                  \
        }                                                                                                              \
        SCAN_P(RPT_, KP_, V_, 0);                                                                                      \
    } while (0)
#define SCAN(RPT_, KP_)                                                                                                \
    do {                                                                                                               \
        if (vec) SCAN_V(RPT_, KP_, true);                                                                              \
        SCAN_V(RPT_, KP_, false);                                                                                      \
    } while (0)
    if (d <= 64) SCAN(4, 16);
    if (narrow) {
        if (d <= 128) SCAN(4, 32);
        SCAN(8, 32);
    }
    if (d <= 128) SCAN(8, 16);
    SCAN(16, 16);
#undef SCAN
#undef SCAN_V
#undef SCAN_P
}

// One token a sequence: gates, recurrence, head norm (norm_w [H * dv]) and gate (gate: [T, H * dv] 32-bit logits, rows of
// ldg, through gate_fn, GATE_*); out: [T, H * dv] in out_dt (rows of no sequence become zeros).  Returns -1, with nothing
// launched, for sizes it does not take.
MOE_API int moe_mlstm_step(const float* proj, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                           const float* i_bias, const float* f_bias, float cap, float q_scale, float* state,
                           long long state_pitch, const float* gate, long long ldg, const float* norm_w, float norm_eps,
                           const int* seq_of_token, const int* cu_seqlens, const int* slots, int num_tokens, int num_seqs,
                           int H, int d, int dv, int gate_fn, void* out, int out_dt, cudaStream_t stream) {
    if (num_seqs <= 0 || num_tokens <= 0) return 0;
    if (!gate || !norm_w || !seq_of_token || !out || ldg < (long long)H * dv || num_seqs > 65535 ||
        mlstm_bad(proj, ld, q_at, k_at, v_at, i_at, f_at, i_bias, f_bias, state, state_pitch, cu_seqlens, slots, H, d, dv, cap))
        return (int)cudaErrorInvalidValue;
    if (dv % 4 || dv > 512 || state_pitch % 4 || !aligned16(state)) return -1;
    const int cg = dv / 4, kp = 256 / cg, units = (d + kp - 1) / kp;
    const size_t smem = ((size_t)2 * ((d + 3) & ~3) + dv + (size_t)kp * dv) * sizeof(float);
    if (units > 32 || smem > 48 * 1024) return -1;
    const MemSeq p{proj, ld, q_at, k_at, v_at, i_at, f_at, i_bias, f_bias, state, state_pitch, cu_seqlens, slots, nullptr,
                   H, d, dv, cap, q_scale, (dv + COPY_COLS - 1) / COPY_COLS};
#define STEP(OT_, U_)                                                                                                  \
    return launch_pdl(mlstm_step_kernel<OT_, U_>, dim3(H, num_seqs), dim3(256), smem, stream, p, gate, ldg, norm_w, norm_eps, \
                      seq_of_token, num_tokens, gate_fn, (OT_*)out)
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
