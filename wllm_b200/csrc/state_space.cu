// A state space with a scalar decay per head and token (Mamba-2): a matrix state S [N, V] per (request, head), 32-bit,
//
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T,    y_t = S_t^T C_t + D_h x_t,    a_t = exp(-exp(A_log_h) dt_t)
//
// B and C are rows of N shared by the heads of a group, x the head's V values.  The recurrence itself is the decayed-state scan of
// linear_attention.cu (q = C, k = B, v = x, with a pair (a - 1, dt) per head and token); here is what stands in front of it
// and behind it, and a chunked form of it for bfloat16 prompts.  Inputs come from one fused projection row z | x | B | C | dt, possibly in
// split-K slabs; what enters the recurrence beside x, B and C is 32-bit.
//
//   wllm_ssd_prepare      the causal convolution of x | B | C along the sequence, channel by channel (`taps` taps, the last weighs the
//                         token itself, inputs in front of the sequence count as zero), its bias, SiLU: one 32-bit row a token; and
//                         dt = softplus(dt + dt_bias) with a - 1 = expm1(-exp(A_log) dt) (a head that forgets slowly has a close to
//                         one, and the rounding of a itself would grow with its memory).  In a step of single tokens it also
//                         shifts the slots' inputs: the thread that read a channel's writes them.  For the chunked form the row goes out in
//                         bfloat16 and the pair is (log a, dt).
//   wllm_ssd_conv_update  the slots' last taps - 1 inputs after this step's tokens, for steps with portions.
//   wllm_ssd_chunks       the recurrence in chunks of 64 tokens on the tensor cores (mma.sync, 32-bit accumulators): with c_t the sum of the
//                         chunk's log a up to t and S the state in front of the chunk,
//                             y_t = exp(c_t) C_t S + sum_(s <= t) (C_t . B_s) exp(c_t - c_s) dt_s x_s
//                             S  <- exp(c_end) S + sum_s B_s (exp(c_end - c_s) dt_s x_s)^T
//                         C, B and x are bfloat16 (outputs of a convolution and SiLU); S stays in 32-bit accumulators from chunk to chunk and,
//                         like the weighted scores and values, enters a product as two bfloat16 pieces (some sixteen bits).
//   wllm_ssd_gate_norm    y = (o + D_h x) silu(z), each of `groups` equal parts of the row divided by its own root mean square,
//                         times a gain, rounded once to the matrix type (the operand of the output projection).
#include "common.cuh"

__device__ __forceinline__ float ss_any(const void* p, int dtype, size_t i) {
    return dtype == WLLM_BF16 ? __bfloat162float(reinterpret_cast<const bf16*>(p)[i]) : reinterpret_cast<const float*>(p)[i];
}
// element i of a row that may come as `parts` 32-bit slabs `stride` elements apart, added in slab order (sixteen loads in flight)
template <bool MULTI>
__device__ __forceinline__ float ss_in(const void* p, int dtype, int parts, size_t stride, size_t i) {
    if (!MULTI || parts == 1) return ss_any(p, dtype, i);
    const float* f = reinterpret_cast<const float*>(p) + i;
    float v = 0.f;
    for (int s0 = 0; s0 < parts; s0 += 16) {
        float part[16];
#pragma unroll
        for (int u = 0; u < 16; ++u) part[u] = s0 + u < parts ? f[(size_t)(s0 + u) * stride] : 0.f;
#pragma unroll
        for (int u = 0; u < 16; ++u)
            if (s0 + u < parts) v = (s0 + u == 0) ? part[u] : v + part[u];
    }
    return v;
}
__device__ __forceinline__ float ss_silu(float z) { return z / (1.0f + expf(-z)); }

constexpr int SS_MAX_TAPS = 16;

// grid (tiles of TT tokens, ceil(C / 256) + 1), 256 threads: a thread a channel, the last row of CTAs the heads' steps and decays.
// TT > 1: the tile's inputs are loaded once and slide through registers (TAPS taps, a template parameter); TT == 1: only the
// inputs that the token's request brings are loaded, the others come from its slot; TAPS == 0: any number of taps.
template <int TT, int TAPS, bool MULTI, typename TO>
__global__ void __launch_bounds__(256)
ssd_prepare_kernel(const void* __restrict__ fused, int in_dtype, int row_stride, int parts, size_t part_stride, int x_off, int dt_off,
                   int n, int C, int H, int any_taps, const void* __restrict__ conv, const void* __restrict__ conv_bias,
                   const void* __restrict__ a_log, const void* __restrict__ dt_bias, int w_dtype, const int* __restrict__ token_req,
                   const int* __restrict__ req_q_start, const int* __restrict__ req_q_len, const int* __restrict__ req_slot,
                   float* __restrict__ conv_state, TO* __restrict__ out, float* __restrict__ pairs, int shift, int logs) {
    pdl_begin();
    const int t0 = blockIdx.x * TT, count = min(TT, n - t0);
    if (blockIdx.y == gridDim.y - 1) {
        for (int idx = threadIdx.x; idx < count * H; idx += blockDim.x) {
            const int t = t0 + idx / H, h = idx % H;
            const float z = ss_in<MULTI>(fused, in_dtype, parts, part_stride, (size_t)t * row_stride + dt_off + h) + ss_any(dt_bias, w_dtype, h);
            const float step = z > 20.f ? z : log1pf(expf(z));
            const float log_a = -expf(ss_any(a_log, w_dtype, h)) * step;
            pairs[((size_t)t * H + h) * 2] = logs ? log_a : expm1f(log_a);
            pairs[((size_t)t * H + h) * 2 + 1] = step;
        }
        return;
    }
    const int ch = blockIdx.y * blockDim.x + threadIdx.x;
    if (ch >= C) return;
    const int taps = TAPS > 0 ? TAPS : any_taps;
    const float bias = conv_bias ? ss_any(conv_bias, w_dtype, ch) : 0.f;
    auto input = [&](int t) { return ss_in<MULTI>(fused, in_dtype, parts, part_stride, (size_t)t * row_stride + x_off + ch); };
    auto weight = [&](int j) { return ss_any(conv, w_dtype, (size_t)ch * taps + (taps - 1 - j)); };       // of the input j tokens back
    if constexpr (TT == 1) {
        const int t = t0, r = token_req[t], i = t - req_q_start[r], slot = req_slot[r];
        const bool keep = shift && slot >= 0 && req_q_len[r] > 0;     // (a row that stands for no token leaves the state alone)
        auto one = [&](int j, float acc) {                          // the oldest input first: one order for every way of cutting
            float x;
            if (i - j >= 0) x = input(t - j);
            else x = slot >= 0 ? conv_state[((size_t)slot * (taps - 1) + (taps - 1 + i - j)) * C + ch] : 0.f;
            // every request brings one token: the input j tokens back is j + 1 back for the next one
            if (keep && j < taps - 1) conv_state[((size_t)slot * (taps - 1) + (taps - 2 - j)) * C + ch] = x;
            return fmaf(weight(j), x, acc);
        };
        float acc = bias;
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = TAPS - 1; j >= 0; --j) acc = one(j, acc);
        } else {
            for (int j = taps - 1; j >= 0; --j) acc = one(j, acc);
        }
        out[(size_t)t * C + ch] = from_f32<TO>(ss_silu(acc));
    } else {
        float w[TAPS], x[TT + TAPS - 1];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = weight(j);
#pragma unroll
        for (int k = 0; k < TT + TAPS - 1; ++k) {
            const int t = t0 - (TAPS - 1) + k;
            x[k] = t >= 0 && t < n ? input(t) : 0.f;
        }
#pragma unroll
        for (int tt = 0; tt < TT; ++tt) {
            if (tt >= count) break;
            const int t = t0 + tt, r = token_req[t], i = t - req_q_start[r];
            float acc = bias;
            if (i >= TAPS - 1) {
#pragma unroll
                for (int j = TAPS - 1; j >= 0; --j) acc = fmaf(w[j], x[tt + TAPS - 1 - j], acc);
            } else {
                const int slot = req_slot[r];
#pragma unroll
                for (int j = TAPS - 1; j >= 0; --j) {
                    float v = x[tt + TAPS - 1 - j];
                    if (i - j < 0) v = slot >= 0 ? conv_state[((size_t)slot * (TAPS - 1) + (TAPS - 1 + i - j)) * C + ch] : 0.f;
                    acc = fmaf(w[j], v, acc);
                }
            }
            out[(size_t)t * C + ch] = from_f32<TO>(ss_silu(acc));
        }
    }
}

// grid (requests, ceil(C / 256)): a thread a channel; the taps - 1 inputs that end at the request's last token of this step
__global__ void __launch_bounds__(256)
ssd_conv_update_kernel(const void* __restrict__ fused, int in_dtype, int row_stride, int parts, size_t part_stride, int x_off, int C,
                       int taps, const int* __restrict__ req_q_start, const int* __restrict__ req_q_len, const int* __restrict__ req_slot,
                       float* __restrict__ conv_state) {
    pdl_begin();
    const int r = blockIdx.x, len = req_q_len[r], slot = req_slot[r];
    const int ch = blockIdx.y * blockDim.x + threadIdx.x, keep = taps - 1, t0 = req_q_start[r];
    if (len <= 0 || slot < 0 || ch >= C) return;
    float* st = conv_state + (size_t)slot * keep * C + ch;
    float vals[SS_MAX_TAPS];
#pragma unroll
    for (int s = 0; s < SS_MAX_TAPS; ++s)
        if (s < keep) {
            const int src = len - keep + s;               // place among this step's tokens; negative: an input kept from before
            vals[s] = src >= 0 ? ss_in<true>(fused, in_dtype, parts, part_stride, (size_t)(t0 + src) * row_stride + x_off + ch)
                               : st[(size_t)(s + len) * C];
        }
#pragma unroll
    for (int s = 0; s < SS_MAX_TAPS; ++s)
        if (s < keep) st[(size_t)s * C] = vals[s];
}

constexpr int SC_Q = 64, SC_VT = 32, SC_THREADS = 256, SC_XP = SC_VT + 8, SC_MP = SC_Q + 8;

__device__ __forceinline__ void sc_cp16(void* dst, const void* src, bool valid) {       // 16 bytes, or zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void sc_cp8(void* dst, const void* src, bool valid) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 8 : 0) : "memory");
}
__device__ __forceinline__ void sc_ldsm4(const bf16* p, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_ldsm4_t(const bf16* p, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two neighbouring values as a high and a low bfloat16 piece each
__device__ __forceinline__ void sc_split(float v0, float v1, __nv_bfloat162& hi, __nv_bfloat162& lo) {
    hi = __floats2bfloat162_rn(v0, v1);
    const float2 h = __bfloat1622float2(hi);
    lo = __floats2bfloat162_rn(v0 - h.x, v1 - h.y);
}

// State rows N = 16 NT.  grid (tiles of 32 value columns, H, requests), 256 threads.  A CTA walks its request's chunks in order; the next
// chunk's rows are on their way while one is worked on.  Warp w holds rows 16 w .. 16 w + 15 of S.  The scores and outputs of a chunk are cut into 4 x 2
// pieces of 16 rows by half the columns.  Tokens behind a request's last read as zeros and change nothing.
template <int NT>
struct ChunkSmem {
    static constexpr int N = 16 * NT, NP = N + 8;
    bf16 B[2][SC_Q][NP], C[2][SC_Q][NP], X[2][SC_Q][SC_XP];
    bf16 M[2][SC_Q][SC_MP];        // the weighted scores: high pieces, low pieces
    bf16 U[2][SC_Q][SC_XP];        // the weighted values
    bf16 S[2][N][SC_XP];           // the state in front of the chunk
    float2 pair[2][SC_Q];          // (log a, dt)
    float cum[SC_Q], ecum[SC_Q], weight[SC_Q];
};

template <int NT>
__global__ void __launch_bounds__(SC_THREADS, 1)
ssd_chunk_kernel(const bf16* __restrict__ xbc, int row_stride, int b_off, int c_off, const float* __restrict__ pairs, float* __restrict__ state,
                 float* __restrict__ out, const int* __restrict__ req_q_start, const int* __restrict__ req_q_len,
                 const int* __restrict__ req_slot, int H, int share, int V) {
    constexpr int N = 16 * NT;
    extern __shared__ __align__(16) unsigned char sc_raw[];
    ChunkSmem<NT>& sm = *reinterpret_cast<ChunkSmem<NT>*>(sc_raw);
    pdl_begin();
    const int r = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * SC_VT;
    const int len = req_q_len[r], slot = req_slot[r];
    if (len <= 0 || slot < 0) return;                      // a request that brings no token
    const int t0 = req_q_start[r], group = h / share;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp & 3, wn = warp >> 2;
    const int frow = lane >> 2, fcol = (lane & 3) * 2;     // this lane's place in an accumulator piece
    float* Sg = state + ((size_t)slot * H + h) * N * V;
    float S[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int row = warp * 16 + frow + (e >> 1) * 8, col = v0 + j * 8 + fcol + (e & 1);
            S[j][e] = (warp < NT && col < V) ? Sg[(size_t)row * V + col] : 0.f;
        }
    auto load = [&](int chunk, int stage) {
        const int first = t0 + chunk * SC_Q, count = min(SC_Q, len - chunk * SC_Q);
        for (int idx = threadIdx.x; idx < SC_Q * (N / 8); idx += SC_THREADS) {
            const int t = idx / (N / 8), c = (idx % (N / 8)) * 8;
            const bool in = t < count;
            const bf16* src = xbc + (size_t)(first + (in ? t : 0)) * row_stride + group * N + c;
            sc_cp16(&sm.B[stage][t][c], src + b_off, in);
            sc_cp16(&sm.C[stage][t][c], src + c_off, in);
        }
        {
            const int t = threadIdx.x >> 2, c = (threadIdx.x & 3) * 8;       // 64 rows of four pieces
            const bool in = t < count && v0 + c < V;
            sc_cp16(&sm.X[stage][t][c], in ? xbc + (size_t)(first + t) * row_stride + h * V + v0 + c : xbc, in);
        }
        if (threadIdx.x < SC_Q) {
            const bool in = threadIdx.x < count;
            sc_cp8(&sm.pair[stage][threadIdx.x], in ? pairs + ((size_t)(first + threadIdx.x) * H + h) * 2 : pairs, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int chunks = (len + SC_Q - 1) / SC_Q;
    load(0, 0);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        const int st = chunk & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (warp < NT) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    __nv_bfloat162 hi, lo;
                    sc_split(S[j][half * 2], S[j][half * 2 + 1], hi, lo);
                    const int row = warp * 16 + frow + half * 8, col = j * 8 + fcol;
                    *reinterpret_cast<__nv_bfloat162*>(&sm.S[0][row][col]) = hi;
                    *reinterpret_cast<__nv_bfloat162*>(&sm.S[1][row][col]) = lo;
                }
        }
        __syncthreads();                                   // the chunk's rows and the state are here; everyone is done with the chunk before
        if (chunk + 1 < chunks) load(chunk + 1, st ^ 1);
        // ---- scores C B^T where some s <= t; the piece that has none sums the logarithms instead
        float G[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) G[j][0] = G[j][1] = G[j][2] = G[j][3] = 0.f;
        if (wn == 0 || wm >= 2) {
#pragma unroll
            for (int k = 0; k < N; k += 16) {
                uint32_t a[4];
                sc_ldsm4(&sm.C[st][wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][k + (lane >> 4) * 8], a);
#pragma unroll
                for (int jj = 0; jj < 2; ++jj) {
                    if (wn * 32 + jj * 16 > wm * 16 + 15) continue;
                    uint32_t b[4];
                    sc_ldsm4(&sm.B[st][wn * 32 + jj * 16 + (lane & 7) + (lane >> 4) * 8][k + ((lane >> 3) & 1) * 8], b);
                    sc_mma(G[2 * jj], a, b[0], b[1]);
                    sc_mma(G[2 * jj + 1], a, b[2], b[3]);
                }
            }
        } else if (wm == 0) {
            const float2 p0 = sm.pair[st][2 * lane], p1 = sm.pair[st][2 * lane + 1];
            float sum = p0.x + p1.x;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float other = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += other;
            }
            float before = __shfl_up_sync(0xffffffffu, sum, 1);
            if (lane == 0) before = 0.f;
            const float all = __shfl_sync(0xffffffffu, sum, 31);
            const float c0 = before + p0.x, c1 = sum;
            sm.cum[2 * lane] = c0;
            sm.cum[2 * lane + 1] = c1;
            sm.ecum[2 * lane] = expf(c0);
            sm.ecum[2 * lane + 1] = expf(c1);
            sm.weight[2 * lane] = expf(all - c0) * p0.y;
            sm.weight[2 * lane + 1] = expf(all - c1) * p1.y;
        }
        __syncthreads();                                   // the sums are here
        // ---- weighted scores and weighted values as two pieces each
        if (wn == 0 || wm >= 2) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int s = wn * 32 + j * 8 + fcol;
                if (wn * 32 + j * 8 > wm * 16 + 15) continue;
                const float cs0 = sm.cum[s], cs1 = sm.cum[s + 1], d0 = sm.pair[st][s].y, d1 = sm.pair[st][s + 1].y;
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int t = wm * 16 + frow + half * 8;
                    const float ct = sm.cum[t];
                    const float m0 = s <= t ? G[j][half * 2] * (expf(ct - cs0) * d0) : 0.f;
                    const float m1 = s + 1 <= t ? G[j][half * 2 + 1] * (expf(ct - cs1) * d1) : 0.f;
                    __nv_bfloat162 hi, lo;
                    sc_split(m0, m1, hi, lo);
                    *reinterpret_cast<__nv_bfloat162*>(&sm.M[0][t][s]) = hi;
                    *reinterpret_cast<__nv_bfloat162*>(&sm.M[1][t][s]) = lo;
                }
            }
        }
        {
            const int s = threadIdx.x >> 2, c = (threadIdx.x & 3) * 8;
            const float w = sm.weight[s];
            const uint4 raw = *reinterpret_cast<const uint4*>(&sm.X[st][s][c]);
            const __nv_bfloat162* x2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
            uint4 hi4, lo4;
            __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&hi4);
            __nv_bfloat162* l2 = reinterpret_cast<__nv_bfloat162*>(&lo4);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(x2[e]);
                sc_split(f.x * w, f.y * w, h2[e], l2[e]);
            }
            *reinterpret_cast<uint4*>(&sm.U[0][s][c]) = hi4;
            *reinterpret_cast<uint4*>(&sm.U[1][s][c]) = lo4;
        }
        // ---- the outputs' share of the state in front of the chunk
        float Y[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) Y[j][0] = Y[j][1] = Y[j][2] = Y[j][3] = 0.f;
#pragma unroll
        for (int k = 0; k < N; k += 16) {
            uint32_t a[4], b[4];
            sc_ldsm4(&sm.C[st][wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][k + (lane >> 4) * 8], a);
#pragma unroll
            for (int p = 1; p >= 0; --p) {
                sc_ldsm4_t(&sm.S[p][k + (lane & 7) + ((lane >> 3) & 1) * 8][wn * 16 + (lane >> 4) * 8], b);
                sc_mma(Y[0], a, b[0], b[1]);
                sc_mma(Y[1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) Y[j][e] *= sm.ecum[wm * 16 + frow + (e >> 1) * 8];
        __syncthreads();                                   // the pieces are here
        // ---- the outputs' share of the chunk's own tokens
        for (int kk = 0; kk <= wm; ++kk) {
            uint32_t b[4];
            sc_ldsm4_t(&sm.X[st][kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][wn * 16 + (lane >> 4) * 8], b);
#pragma unroll
            for (int p = 1; p >= 0; --p) {
                uint32_t a[4];
                sc_ldsm4(&sm.M[p][wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][kk * 16 + (lane >> 4) * 8], a);
                sc_mma(Y[0], a, b[0], b[1]);
                sc_mma(Y[1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = chunk * SC_Q + wm * 16 + frow + half * 8, col = v0 + wn * 16 + j * 8 + fcol;
                if (t < len && col < V)                    // (V in steps of 8: a pair of columns lies inside or outside)
                    *reinterpret_cast<float2*>(out + ((size_t)(t0 + t) * H + h) * V + col) = make_float2(Y[j][half * 2], Y[j][half * 2 + 1]);
            }
        // ---- the state behind the chunk
        if (warp < NT) {
            const float fade = sm.ecum[SC_Q - 1];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] *= fade;
#pragma unroll
            for (int kk = 0; kk < SC_Q / 16; ++kk) {
                uint32_t a[4];
                sc_ldsm4_t(&sm.B[st][kk * 16 + (lane & 7) + (lane >> 4) * 8][warp * 16 + ((lane >> 3) & 1) * 8], a);
#pragma unroll
                for (int p = 1; p >= 0; --p)
#pragma unroll
                    for (int jj = 0; jj < 2; ++jj) {
                        uint32_t b[4];
                        sc_ldsm4_t(&sm.U[p][kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][jj * 16 + (lane >> 4) * 8], b);
                        sc_mma(S[2 * jj], a, b[0], b[1]);
                        sc_mma(S[2 * jj + 1], a, b[2], b[3]);
                    }
            }
        }
    }
    if (warp < NT) {
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = warp * 16 + frow + half * 8, col = v0 + j * 8 + fcol;
                if (col < V) *reinterpret_cast<float2*>(Sg + (size_t)row * V + col) = make_float2(S[j][half * 2], S[j][half * 2 + 1]);
            }
    }
}

// grid (tokens, groups): the part of the row in shared memory between its sum of squares (a block sum in a fixed order) and the scaling
template <typename TO, bool MULTI>
__global__ void ssd_gate_norm_kernel(const float* __restrict__ o, const void* __restrict__ x, int x_dtype, size_t x_stride, const void* __restrict__ skip,
                                     const void* __restrict__ fused, int in_dtype, int row_stride, int parts, size_t part_stride, int z_off,
                                     const void* __restrict__ w, int w_dtype, float eps, TO* __restrict__ out, int inner, int V, int part) {
    extern __shared__ float ss_row[];
    __shared__ float scratch[32];
    pdl_begin();
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* orow = o + (size_t)t * inner + c0;
    const size_t xrow = (size_t)t * x_stride + c0;
    const size_t zrow = (size_t)t * row_stride + z_off + c0;
    float ss = 0.f;
    for (int c = threadIdx.x; c < part; c += blockDim.x) {
        const float z = ss_in<MULTI>(fused, in_dtype, parts, part_stride, zrow + c);
        const float y = fmaf(ss_any(skip, w_dtype, (c0 + c) / V), ss_any(x, x_dtype, xrow + c), orow[c]) * ss_silu(z);
        ss_row[c] = y;
        ss = fmaf(y, y, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    TO* dst = out + (size_t)t * inner + c0;
    for (int c = threadIdx.x; c < part; c += blockDim.x) dst[c] = from_f32<TO>((ss_row[c] * inv) * ss_any(w, w_dtype, c0 + c));
}

// The same for bfloat16 rows whose parts and heads come in steps of 4 elements: 16-byte loads of o and x, 8-byte loads of the gate and
// the gain, 8-byte stores.
template <typename TX>
__device__ __forceinline__ float4 ss_load4(const TX* p);
template <> __device__ __forceinline__ float4 ss_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 ss_load4<bf16>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

template <typename TX>
__global__ void ssd_gate_norm_vec_kernel(const float* __restrict__ o, const TX* __restrict__ x, size_t x_stride, const bf16* __restrict__ skip,
                                         const bf16* __restrict__ fused, int row_stride, int z_off, const bf16* __restrict__ w, float eps,
                                         bf16* __restrict__ out, int inner, int V, int part) {
    extern __shared__ float ss_row[];
    __shared__ float scratch[32];
    pdl_begin();
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* orow = o + (size_t)t * inner + c0;
    const TX* xrow = x + (size_t)t * x_stride + c0;
    const bf16* zrow = fused + (size_t)t * row_stride + z_off + c0;
    float ss = 0.f;
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
        const float4 o4 = ss_load4(orow + c), x4 = ss_load4(xrow + c), z4 = ss_load4(zrow + c);
        const float d = __bfloat162float(skip[(c0 + c) / V]);
        float4 y;
        y.x = fmaf(d, x4.x, o4.x) * ss_silu(z4.x); y.y = fmaf(d, x4.y, o4.y) * ss_silu(z4.y);
        y.z = fmaf(d, x4.z, o4.z) * ss_silu(z4.z); y.w = fmaf(d, x4.w, o4.w) * ss_silu(z4.w);
        *reinterpret_cast<float4*>(ss_row + c) = y;
        ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    bf16* dst = out + (size_t)t * inner + c0;
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
        const float4 y = *reinterpret_cast<const float4*>(ss_row + c), w4 = ss_load4(w + c0 + c);
        const __nv_bfloat162 a = __floats2bfloat162_rn((y.x * inv) * w4.x, (y.y * inv) * w4.y);
        const __nv_bfloat162 b = __floats2bfloat162_rn((y.z * inv) * w4.z, (y.w * inv) * w4.w);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&a);
        packed.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(dst + c) = packed;
    }
}

// fused [n, W] (or `parts` 32-bit slabs): x | B | C at x_off (C columns), dt at dt_off [H]; conv [C, taps], conv_bias [C] (may be null),
// a_log, dt_bias [H] of one element type; conv_state [slots, taps - 1, C]; out [n, C] (32-bit, or bfloat16: then pairs holds (log a, dt)),
// pairs [n, H, 2] = (a - 1, dt), 32-bit.
// shift: every request of the step brings at most one token, and conv_state is brought up to date here.
WLLM_API int wllm_ssd_prepare(const void* fused, int in_dtype, int row_stride, int parts, long long part_stride, int x_off, int dt_off, int n,
                              int C, int H, int taps, const void* conv, const void* conv_bias, const void* a_log, const void* dt_bias,
                              int w_dtype, const int* token_req, const int* req_q_start, const int* req_q_len, const int* req_slot,
                              float* conv_state, void* out, int out_dtype, float* pairs, int shift, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (C <= 0 || H <= 0 || taps < 1 || taps > SS_MAX_TAPS || parts < 1 || (taps > 1 && conv_state == nullptr)) return WLLM_BAD_SIZE;
    if ((in_dtype != WLLM_BF16 && in_dtype != WLLM_F32) || (w_dtype != WLLM_BF16 && w_dtype != WLLM_F32)) return WLLM_BAD_DTYPE;
    if (out_dtype != WLLM_BF16 && out_dtype != WLLM_F32) return WLLM_BAD_DTYPE;
    const int rows = (C + 255) / 256 + 1;
    if (rows > 65535) return WLLM_BAD_SIZE;
#define PREP2(TT, TAPS, M, TO) wllm_launch(ssd_prepare_kernel<TT, TAPS, M, TO>, dim3((n + TT - 1) / TT, rows), 256, 0, stream, fused, in_dtype, row_stride, \
        parts, (size_t)part_stride, x_off, dt_off, n, C, H, taps, conv, conv_bias, a_log, dt_bias, w_dtype, token_req, req_q_start, req_q_len, \
        req_slot, conv_state, (TO*)out, pairs, shift, out_dtype == WLLM_BF16 ? 1 : 0)
#define PREP(TT, TAPS, M) (out_dtype == WLLM_BF16 ? PREP2(TT, TAPS, M, bf16) : PREP2(TT, TAPS, M, float))
    if (parts == 1 && n >= 256 && !shift) {      // many tokens: a tile's inputs are loaded once
        if (taps == 2) return PREP(8, 2, false);
        if (taps == 3) return PREP(8, 3, false);
        if (taps == 4) return PREP(8, 4, false);
    }
    if (taps == 4) return parts > 1 ? PREP(1, 4, true) : PREP(1, 4, false);
    return parts > 1 ? PREP(1, 0, true) : PREP(1, 0, false);
#undef PREP
#undef PREP2
}

template <int NT>
static int launch_chunks(const bf16* xbc, int row_stride, int b_off, int c_off, const float* pairs, float* state, float* out, const int* req_q_start,
                         const int* req_q_len, const int* req_slot, int requests, int H, int share, int V, cudaStream_t stream) {
    static bool raised = false;
    if (!raised) {
        const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(ChunkSmem<NT>));
        if (e != cudaSuccess) return 1000 + (int)e;
        raised = true;
    }
    return wllm_launch(ssd_chunk_kernel<NT>, dim3((V + SC_VT - 1) / SC_VT, H, requests), SC_THREADS, sizeof(ChunkSmem<NT>), stream, xbc, row_stride, b_off,
                       c_off, pairs, state, out, req_q_start, req_q_len, req_slot, H, share, V);
}

// xbc [n, ..] bfloat16 with rows row_stride apart: x from column 0 [H * V], B from b_off and C from c_off [H / share * N each]; pairs [n, H, 2] =
// (log a, dt); state [slots, H, N, V]; out [n, H, V].  N in steps of 16 up to 128, V and the row's places in steps of 8.
WLLM_API int wllm_ssd_chunks(const void* xbc, int row_stride, int b_off, int c_off, const float* pairs, float* state, float* out,
                             const int* req_q_start, const int* req_q_len, const int* req_slot, int requests, int H, int share, int N, int V,
                             cudaStream_t stream) {
    if (requests <= 0) return WLLM_OK;
    if (H <= 0 || H > 65535 || requests > 65535 || share < 1 || H % share != 0 || N < 16 || N > 128 || N % 16 != 0 || V < 8 || V % 8 != 0) return WLLM_BAD_SIZE;
    if (row_stride % 8 != 0 || b_off % 8 != 0 || c_off % 8 != 0 || ((uintptr_t)xbc & 15) || ((uintptr_t)pairs & 7) || ((uintptr_t)state & 7) ||
        ((uintptr_t)out & 7))
        return WLLM_BAD_ALIGN;
#define GO(NT) case NT: return launch_chunks<NT>((const bf16*)xbc, row_stride, b_off, c_off, pairs, state, out, req_q_start, req_q_len, req_slot, \
                                                 requests, H, share, V, stream)
    switch (N / 16) { GO(1); GO(2); GO(3); GO(4); GO(5); GO(6); GO(7); GO(8); }
#undef GO
    return WLLM_BAD_SIZE;
}

WLLM_API int wllm_ssd_conv_update(const void* fused, int in_dtype, int row_stride, int parts, long long part_stride, int x_off, int C, int taps,
                                  const int* req_q_start, const int* req_q_len, const int* req_slot, int requests, float* conv_state,
                                  cudaStream_t stream) {
    if (requests <= 0 || taps <= 1) return WLLM_OK;
    if (C <= 0 || taps > SS_MAX_TAPS || parts < 1 || conv_state == nullptr || (C + 255) / 256 > 65535) return WLLM_BAD_SIZE;
    if (in_dtype != WLLM_BF16 && in_dtype != WLLM_F32) return WLLM_BAD_DTYPE;
    return wllm_launch(ssd_conv_update_kernel, dim3(requests, (C + 255) / 256), 256, 0, stream, fused, in_dtype, row_stride, parts,
                       (size_t)part_stride, x_off, C, taps, req_q_start, req_q_len, req_slot, conv_state);
}

// o [n, inner] 32-bit, x [n, ..] of either type with rows x_stride apart; skip [inner / V] and w [inner] of one element type; the gate z at z_off of fused
WLLM_API int wllm_ssd_gate_norm(const float* o, const void* x, int x_dtype, long long x_stride, const void* skip, const void* fused, int in_dtype,
                                int row_stride, int parts, long long part_stride, int z_off, const void* w, int w_dtype, float eps, void* out,
                                int out_dtype, int n, int inner, int V, int groups, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (inner <= 0 || V <= 0 || inner % V != 0 || groups < 1 || groups > 65535 || inner % groups != 0 || parts < 1 || x_stride < inner)
        return WLLM_BAD_SIZE;
    if ((in_dtype != WLLM_BF16 && in_dtype != WLLM_F32) || (w_dtype != WLLM_BF16 && w_dtype != WLLM_F32) || (x_dtype != WLLM_BF16 && x_dtype != WLLM_F32))
        return WLLM_BAD_DTYPE;
    const int part = inner / groups;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 192 * 1024) return WLLM_BAD_SIZE;
    static bool raised = false;
    if (!raised && smem > 48 * 1024) {
        cudaError_t e = cudaSuccess;
#define RAISE(K) if (e == cudaSuccess) e = cudaFuncSetAttribute(K, cudaFuncAttributeMaxDynamicSharedMemorySize, 192 * 1024)
        RAISE((ssd_gate_norm_kernel<bf16, true>)); RAISE((ssd_gate_norm_kernel<bf16, false>));
        RAISE((ssd_gate_norm_kernel<float, true>)); RAISE((ssd_gate_norm_kernel<float, false>));
        RAISE(ssd_gate_norm_vec_kernel<float>); RAISE(ssd_gate_norm_vec_kernel<bf16>);
#undef RAISE
        if (e != cudaSuccess) return 1000 + (int)e;
        raised = true;
    }
    const dim3 grid(n, groups);
    if (parts == 1 && in_dtype == WLLM_BF16 && w_dtype == WLLM_BF16 && out_dtype == WLLM_BF16 && part % 4 == 0 && V % 4 == 0 && x_stride % 4 == 0 &&
        row_stride % 4 == 0 && z_off % 4 == 0 && !(((uintptr_t)o | (uintptr_t)x) & 15) && !(((uintptr_t)fused | (uintptr_t)w | (uintptr_t)out) & 7)) {
        const int threads = part >= 2048 ? 256 : (part >= 512 ? 128 : 64);
#define VEC(TX) wllm_launch(ssd_gate_norm_vec_kernel<TX>, grid, threads, smem, stream, o, (const TX*)x, (size_t)x_stride, (const bf16*)skip, \
                            (const bf16*)fused, row_stride, z_off, (const bf16*)w, eps, (bf16*)out, inner, V, part)
        return x_dtype == WLLM_BF16 ? VEC(bf16) : VEC(float);
#undef VEC
    }
    const int threads = part >= 2048 ? 512 : (part >= 512 ? 256 : 128);
#define GATE(TO, M) wllm_launch(ssd_gate_norm_kernel<TO, M>, grid, threads, smem, stream, o, x, x_dtype, (size_t)x_stride, skip, fused, in_dtype, row_stride, \
        parts, (size_t)part_stride, z_off, w, w_dtype, eps, (TO*)out, inner, V, part)
    if (out_dtype == WLLM_BF16) return parts > 1 ? GATE(bf16, true) : GATE(bf16, false);
    if (out_dtype == WLLM_F32) return parts > 1 ? GATE(float, true) : GATE(float, false);
#undef GATE
    return WLLM_BAD_DTYPE;
}
