// A real-gated linear recurrent unit behind a short convolution, channel by channel:
//
//     x = in_x + b_x                       u_t = b_c + sum_j taps[:, T - 1 - j] x_(t - j)        (T taps that look back only)
//     r = sigmoid(R_b u_b + ..), i = sigmoid(I_b u_b + ..)      for every of B equal blocks u_b of the channels
//     log a = -c r softplus(lam);          S_t = a S_(t-1) + sqrt(1 - a^2) i u;                  out_t = S_t gelu_tanh(in_y + b_y)
//
// in_y and in_x are columns of one projection row (possibly still in split-K slabs).  The convolution, the gates and the
// recurrence are 32-bit.  A channel that forgets slowly has a close to one, and what counts is how far it is from one: a - 1 is
// carried instead of a (e = expm1(log a), S + (e S + b), 1 - a^2 = -e (2 + e)), so that its error is relative to itself and does
// not grow with the memory.  The state S [W] and the last inputs x of the convolution live in the cache manager's state slots.  The
// kept inputs are a ring of T rows: the input of position p lies in row p mod T, so a step of single tokens reads the rows of
// the T - 1 positions before and writes its own without meeting another CTA's reads.  A position before the start counts as zero.
//
//   wllm_rglru_gates   a step's tokens: convolution and gates, (a - 1, sqrt(1 - a^2) i u) as pairs [n, W, 2].  Two forms: the block
//                      maps on the tensor cores (mma.sync, bfloat16 maps: u in two bfloat16 pieces, high and low, so that the product
//                      keeps some sixteen bits of u), and plain 32-bit chains (32-bit maps, sizes in no step of 8).
//   wllm_rglru_conv    many tokens, bfloat16 maps: the convolution alone, u as its two pieces in the layout that the grouped
//                      tensor-memory product (gemm_bf16_tc.cu) reads: a group a block, rows [high | low] of 2 s elements, times the
//                      block's rows [R R; I I] gives both gates' sums in 32-bit.  It writes that product's table of row tiles too.
//   wllm_rglru_scan    the recurrence over every request's tokens from and to its slot, the output gate, and the slot's kept
//                      inputs, from the pairs or from the gates' sums and u's pieces.  Short portions: a thread a channel walks the
//                      tokens.  Long ones: 32 runs of 4 tokens at a time; a run's decay product and end state from zero come first,
//                      then its true start state from the runs before it, then its outputs; all of it from registers, so that
//                      everything is read once, and the next tokens' values are on their way meanwhile.
//   wllm_rglru_step    both at once for a step in which no request brings more than one token (decoding).
#include "common.cuh"

__device__ __forceinline__ float rg_any(const void* p, int dtype, size_t i) {
    return dtype == WLLM_BF16 ? __bfloat162float(reinterpret_cast<const bf16*>(p)[i]) : reinterpret_cast<const float*>(p)[i];
}
// element i of a row that may come as `parts` 32-bit slabs `stride` elements apart, added in slab order (eight loads in flight)
__device__ __forceinline__ float rg_in(const void* p, int dtype, int parts, size_t stride, size_t i) {
    if (parts == 1) return rg_any(p, dtype, i);
    const float* f = reinterpret_cast<const float*>(p) + i;
    float v = 0.f;
    for (int s0 = 0; s0 < parts; s0 += 8) {
        float part[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) part[u] = s0 + u < parts ? f[(size_t)(s0 + u) * stride] : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (s0 + u < parts) v = (s0 + u == 0) ? part[u] : v + part[u];
    }
    return v;
}
// eight neighbouring elements (a bfloat16 tensor, or 32-bit slabs); 16-byte aligned
__device__ __forceinline__ void rg_in8(const void* p, int dtype, int parts, size_t stride, size_t i, float (&v)[8]) {
    if (dtype == WLLM_BF16) {
        const uint4 raw = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p) + i);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h2[e]); v[2 * e] = f.x; v[2 * e + 1] = f.y; }
        return;
    }
    const float* f = reinterpret_cast<const float*>(p) + i;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = 0.f;
    for (int s0 = 0; s0 < parts; s0 += 4) {
        float4 a[4], b[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            a[u] = b[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (s0 + u < parts) {
                a[u] = *reinterpret_cast<const float4*>(f + (size_t)(s0 + u) * stride);
                b[u] = *reinterpret_cast<const float4*>(f + (size_t)(s0 + u) * stride + 4);
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (s0 + u < parts) {
                v[0] += a[u].x; v[1] += a[u].y; v[2] += a[u].z; v[3] += a[u].w;
                v[4] += b[u].x; v[5] += b[u].y; v[6] += b[u].z; v[7] += b[u].w;
            }
    }
}
__device__ __forceinline__ void rg_f8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float rg_gelu_tanh(float x) {
    const float k = 0.7978845608028654f;  // sqrt(2/pi)
    return 0.5f * x * (1.0f + tanhf(k * (x + 0.044715f * x * x * x)));
}

// the step's projection and what goes with it
struct RgInput {
    const void* fused;        // [n, row] or `parts` slabs `part_stride` elements apart
    int dtype, row_stride, parts;
    size_t part_stride;
    int y_off, x_off;         // first columns of in_y and in_x
    const float* x_bias;      // [W]
    const float* y_bias;      // [W]
    const float* taps;        // [T][W]: row j weighs the input of T - 1 - j positions before
    const float* conv_bias;   // [W]
    int T, W;
    const int* positions;
    const int* token_req;
    const int* req_q_start;
    const int* req_slot;
    float* ring;              // [slots][T][W]
};
// gates' parameters
struct RgGates {
    const void* ra;           // B blocks of s rows of s elements ([out, in]), `pitch` elements from row to row, `block` from block to block
    const void* ri;
    int w_dtype, pitch;
    size_t block;
    const float* ra_bias;     // [W]
    const float* ri_bias;
    const float* rate;        // [W] c softplus(lam): log a = -rate r
    int B, s;
};

// x (with its bias) of the token j places before token t of its request
__device__ __forceinline__ float rg_x(const RgInput& in, int t, int i, int slot, int pos, int j, int c) {
    if (pos - j < 0) return 0.f;
    if (i - j >= 0) return rg_in(in.fused, in.dtype, in.parts, in.part_stride, (size_t)(t - j) * in.row_stride + in.x_off + c) + in.x_bias[c];
    return in.ring[((size_t)slot * in.T + (pos - j) % in.T) * in.W + c];
}
__device__ __forceinline__ float rg_conv(const RgInput& in, int t, int c) {
    const int r = in.token_req[t], i = t - in.req_q_start[r], slot = max(in.req_slot[r], 0), pos = in.positions[t];
    float u = in.conv_bias[c];
    for (int j = in.T - 1; j >= 0; --j)        // the oldest input first: one order for every way of cutting
        u = fmaf(in.taps[(size_t)(in.T - 1 - j) * in.W + c], rg_x(in, t, i, slot, pos, j, c), u);
    return u;
}
// eight neighbouring channels
__device__ __forceinline__ void rg_conv8(const RgInput& in, int t, int i, int slot, int pos, int c, float (&u)[8]) {
    float xb[8];
    rg_f8(in.conv_bias + c, u);
    rg_f8(in.x_bias + c, xb);
    for (int j = in.T - 1; j >= 0; --j) {
        if (pos - j < 0) continue;
        float x[8], w[8];
        if (i - j >= 0) {
            rg_in8(in.fused, in.dtype, in.parts, in.part_stride, (size_t)(t - j) * in.row_stride + in.x_off + c, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] += xb[e];
        } else {
            rg_f8(in.ring + ((size_t)slot * in.T + (pos - j) % in.T) * in.W + c, x);
        }
        rg_f8(in.taps + (size_t)(in.T - 1 - j) * in.W + c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] = fmaf(w[e], x[e], u[e]);
    }
}
// (a - 1, sqrt(1 - a^2) i u) from the gates' sums
__device__ __forceinline__ float2 rg_pair(const RgGates& g, int c, float zr, float zi, float u) {
    const float r = rg_sigmoid(zr + g.ra_bias[c]), i = rg_sigmoid(zi + g.ri_bias[c]);
    const float e = expm1f(-g.rate[c] * r);
    return make_float2(e, sqrtf(-e * (2.0f + e)) * (i * u));
}
// one step of the recurrence from such a pair
__device__ __forceinline__ float rg_advance(float S, float2 p) { return S + fmaf(p.x, S, p.y); }

// ---------------------------------------------------------------------------------------------------
// gates, plain: grid (blocks of channels x tiles of 32 of their channels, tiles of 32 tokens), 256 threads; thread (ty, tx) of
// 16 x 16 owns tokens ty, ty + 16 and channels tx, tx + 16; a gate's sum is one ascending chain over the block's channels
// ---------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
rglru_gates_plain_kernel(RgInput in, RgGates g, int n, float2* __restrict__ ab) {
    constexpr int TM = 32, TN = 32, TK = 16;
    __shared__ float Us[TK][TM + 1], Wr[TK][TN + 1], Wi[TK][TN + 1];
    pdl_begin();
    const int tiles = (g.s + TN - 1) / TN, b = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * TN, t0 = blockIdx.y * TM;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, base = b * g.s;
    float acc[2][2][2] = {};
    for (int k0 = 0; k0 < g.s; k0 += TK) {
        for (int idx = threadIdx.x; idx < TM * TK; idx += 256) {
            const int tt = idx / TK, k = idx % TK;
            Us[k][tt] = (t0 + tt < n && k0 + k < g.s) ? rg_conv(in, t0 + tt, base + k0 + k) : 0.f;
        }
        for (int idx = threadIdx.x; idx < TN * TK; idx += 256) {
            const int c = idx / TK, k = idx % TK;
            const bool ok = col0 + c < g.s && k0 + k < g.s;
            const size_t at = b * g.block + (size_t)(col0 + c) * g.pitch + k0 + k;
            Wr[k][c] = ok ? rg_any(g.ra, g.w_dtype, at) : 0.f;
            Wi[k][c] = ok ? rg_any(g.ri, g.w_dtype, at) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; ++k)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float u = Us[k][ty + 16 * i];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    acc[0][i][j] = fmaf(u, Wr[k][tx + 16 * j], acc[0][i][j]);
                    acc[1][i][j] = fmaf(u, Wi[k][tx + 16 * j], acc[1][i][j]);
                }
            }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = t0 + ty + 16 * i, cc = col0 + tx + 16 * j;
            if (t >= n || cc >= g.s) continue;
            ab[(size_t)t * in.W + base + cc] = rg_pair(g, base + cc, acc[0][i][j], acc[1][i][j], rg_conv(in, t, base + cc));
        }
}

// ---------------------------------------------------------------------------------------------------
// gates on the tensor cores: grid (blocks x tiles of 64 channels, tiles of 64 tokens), 256 threads (2 x 4 warps: 32 tokens by 16
// channels of both gates each).  The block's channels come in runs of 32: the convolution of 64 tokens (eight channels a
// thread) goes to shared memory as a high and a low bfloat16 piece, the maps' rows through cp.async; two buffers.
// ---------------------------------------------------------------------------------------------------
constexpr int RG_TM = 64, RG_TN = 64, RG_TK = 32, RG_PITCH = RG_TK + 8;
constexpr int RG_UPITCH = RG_TN + 1;
struct RgSmem {
    bf16 hi[2][RG_TM][RG_PITCH];
    bf16 lo[2][RG_TM][RG_PITCH];
    bf16 w[2][2 * RG_TN][RG_PITCH];
    float u[RG_TM][RG_UPITCH];           // the tile's own channels, 32-bit
};

__device__ __forceinline__ void rg_cp16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void rg_ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rg_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two 32-bit numbers as a pair of bfloat16 pieces each: v = high + low up to some 2^-17 of v
__device__ __forceinline__ void rg_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 back = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - back.x, y - back.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

__global__ void __launch_bounds__(256)
rglru_gates_mma_kernel(RgInput in, RgGates g, int n, float2* __restrict__ ab) {
    extern __shared__ __align__(16) unsigned char rg_smem[];
    RgSmem& sm = *reinterpret_cast<RgSmem*>(rg_smem);
    pdl_launch_dependents();
    const int tiles = (g.s + RG_TN - 1) / RG_TN, b = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * RG_TN, t0 = blockIdx.y * RG_TM;
    const int base = b * g.s, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // the maps' rows: 128 rows (16 of R and 16 of I for every of the four warp columns) of 32 elements, two 16-byte pieces a thread
    const int w_piece = threadIdx.x & 3;
    const bf16* w_src[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = (threadIdx.x >> 2) + 64 * h, col = col0 + 16 * (r >> 5) + (r & 15);
        w_src[h] = col < g.s ? reinterpret_cast<const bf16*>((r >> 4) & 1 ? g.ri : g.ra) + b * g.block + (size_t)col * g.pitch : nullptr;
    }
    auto load_w = [&](int kb, int buf) {
        const int k = kb * RG_TK + w_piece * 8;
#pragma unroll
        for (int h = 0; h < 2; ++h)
            rg_cp16((uint32_t)__cvta_generic_to_shared(&sm.w[buf][(threadIdx.x >> 2) + 64 * h][w_piece * 8]), w_src[h] ? w_src[h] + k : (const bf16*)g.ra,
                    w_src[h] != nullptr && k < g.s);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_w(0, 0);                                   // (weights: written by no kernel of the step)
    pdl_wait();
    // the convolution: a token and eight channels a thread
    const int u_tok = threadIdx.x >> 2, u_ch = (threadIdx.x & 3) * 8, t = t0 + u_tok;
    int i = 0, slot = 0, pos = 0;
    if (t < n) {
        const int r = in.token_req[t];
        i = t - in.req_q_start[r];
        slot = max(in.req_slot[r], 0);
        pos = in.positions[t];
    }
    auto make_u = [&](int kb, int buf) {
        const int k = kb * RG_TK + u_ch;
        float u[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] = 0.f;
        if (t < n && k < g.s) rg_conv8(in, t, i, slot, pos, base + k, u);
        uint4 hi, lo;
        rg_split2(u[0], u[1], hi.x, lo.x); rg_split2(u[2], u[3], hi.y, lo.y);
        rg_split2(u[4], u[5], hi.z, lo.z); rg_split2(u[6], u[7], hi.w, lo.w);
        *reinterpret_cast<uint4*>(&sm.hi[buf][u_tok][u_ch]) = hi;
        *reinterpret_cast<uint4*>(&sm.lo[buf][u_tok][u_ch]) = lo;
        if (k >= col0 && k < col0 + RG_TN) {
#pragma unroll
            for (int e = 0; e < 8; ++e) sm.u[u_tok][k - col0 + e] = u[e];
        }
    };
    const int wm = warp & 1, wn = warp >> 1;
    float acc[2][4][4];
#pragma unroll
    for (int mi = 0; mi < 2; ++mi)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[mi][j][0] = acc[mi][j][1] = acc[mi][j][2] = acc[mi][j][3] = 0.f;
    const int kblocks = (g.s + RG_TK - 1) / RG_TK;
    make_u(0, 0);
    for (int kb = 0; kb < kblocks; ++kb) {
        const int buf = kb & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                            // block kb is here for everyone; the other buffer is free
        if (kb + 1 < kblocks) { load_w(kb + 1, buf ^ 1); make_u(kb + 1, buf ^ 1); }
#pragma unroll
        for (int kk = 0; kk < RG_TK / 16; ++kk) {
            uint32_t ah[2][4], al[2][4], bw[2][4];
#pragma unroll
            for (int mi = 0; mi < 2; ++mi) {
                const int row = wm * 32 + mi * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, col = kk * 16 + (lane >> 4) * 8;
                rg_ldsm4((uint32_t)__cvta_generic_to_shared(&sm.hi[buf][row][col]), ah[mi]);
                rg_ldsm4((uint32_t)__cvta_generic_to_shared(&sm.lo[buf][row][col]), al[mi]);
            }
#pragma unroll
            for (int nj = 0; nj < 2; ++nj)
                rg_ldsm4((uint32_t)__cvta_generic_to_shared(&sm.w[buf][wn * 32 + nj * 16 + (lane & 7) + (lane >> 4) * 8][kk * 16 + ((lane >> 3) & 1) * 8]), bw[nj]);
#pragma unroll
            for (int mi = 0; mi < 2; ++mi)
#pragma unroll
                for (int nj = 0; nj < 2; ++nj) {
                    rg_mma(acc[mi][2 * nj], al[mi], bw[nj][0], bw[nj][1]);
                    rg_mma(acc[mi][2 * nj + 1], al[mi], bw[nj][2], bw[nj][3]);
                    rg_mma(acc[mi][2 * nj], ah[mi], bw[nj][0], bw[nj][1]);
                    rg_mma(acc[mi][2 * nj + 1], ah[mi], bw[nj][2], bw[nj][3]);
                }
        }
    }
    // columns 16 wn .. + 15: acc[mi][0 / 1] hold R's sums of the first and second eight of them, acc[mi][2 / 3] I's
#pragma unroll
    for (int mi = 0; mi < 2; ++mi)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = wm * 32 + mi * 16 + (lane >> 2) + half * 8;
            if (t0 + row >= n) continue;
#pragma unroll
            for (int ni = 0; ni < 2; ++ni) {
                const int cc = 16 * wn + 8 * ni + (lane & 3) * 2;
                if (col0 + cc >= g.s) continue;     // (s is a multiple of 8: both columns or none)
                const int c = base + col0 + cc;
                const float2 p = rg_pair(g, c, acc[mi][ni][half * 2], acc[mi][ni + 2][half * 2], sm.u[row][cc]);
                const float2 q = rg_pair(g, c + 1, acc[mi][ni][half * 2 + 1], acc[mi][ni + 2][half * 2 + 1], sm.u[row][cc + 1]);
                *reinterpret_cast<float4*>(ab + (size_t)(t0 + row) * in.W + c) = make_float4(p.x, p.y, q.x, q.y);
            }
        }
}

// the convolution alone: grid (tiles of 4 tokens, tiles of 512 channels), 256 threads = 4 tokens by 64 runs of eight channels.
// uv [B][n][2 s]; tiles (null: none): the table of row tiles of `tile_rows` rows of one block each
__global__ void __launch_bounds__(256, 3)
rglru_conv_kernel(RgInput in, int n, int B, int s, bf16* __restrict__ uv, int* __restrict__ tiles, int tile_rows) {
    pdl_begin();
    if (tiles != nullptr && blockIdx.x == 0 && blockIdx.y == 0) {
        const int per = (n + tile_rows - 1) / tile_rows;
        for (int i = threadIdx.x; i < B * per; i += blockDim.x) {
            const int b = i / per, k = i % per;
            tiles[1 + 3 * i] = b;
            tiles[2 + 3 * i] = b * n + k * tile_rows;
            tiles[3 + 3 * i] = min(tile_rows, n - k * tile_rows);
        }
        if (threadIdx.x == 0) tiles[0] = B * per;
    }
    const int t = blockIdx.x * 4 + (threadIdx.x >> 6), c = (blockIdx.y * 64 + (threadIdx.x & 63)) * 8;
    if (t >= n || c >= in.W) return;
    const int r = in.token_req[t];
    float u[8];
    rg_conv8(in, t, t - in.req_q_start[r], max(in.req_slot[r], 0), in.positions[t], c, u);
    uint4 hi, lo;
    rg_split2(u[0], u[1], hi.x, lo.x); rg_split2(u[2], u[3], hi.y, lo.y);
    rg_split2(u[4], u[5], hi.z, lo.z); rg_split2(u[6], u[7], hi.w, lo.w);
    bf16* dst = uv + ((size_t)(c / s) * n + t) * 2 * s + c % s;          // (s is a multiple of 8: the eight channels share a block)
    *reinterpret_cast<uint4*>(dst) = hi;
    *reinterpret_cast<uint4*>(dst + s) = lo;
}

// ---------------------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------------------
// where the recurrence finds a token's pair: made already, or the gates' sums z [B][n][2 s] (R's s, then I's) and u's pieces
struct RgPairs {
    const float2* ab;
    const float* z;
    const bf16* uv;
    int n, s;
};
template <bool MADE>
__device__ __forceinline__ float2 rg_pair_at(const RgPairs& src, const RgGates& g, int W, int t, int c) {
    if (MADE) return src.ab[(size_t)t * W + c];
    const size_t at = ((size_t)(c / src.s) * src.n + t) * 2 * src.s + c % src.s;
    return rg_pair(g, c, src.z[at], src.z[at + src.s], __bfloat162float(src.uv[at]) + __bfloat162float(src.uv[at + src.s]));
}
// the newest inputs of the convolution after this step: rows of the ring (positions base + len - T .. base + len - 1)
__device__ __forceinline__ void rg_keep_inputs(const RgInput& in, int t0, int len, int slot, int first_pos, int c) {
    for (int k = max(0, len - in.T); k < len; ++k)
        in.ring[((size_t)slot * in.T + (first_pos + k) % in.T) * in.W + c] =
            rg_in(in.fused, in.dtype, in.parts, in.part_stride, (size_t)(t0 + k) * in.row_stride + in.x_off + c) + in.x_bias[c];
}
__device__ __forceinline__ float rg_y(const RgInput& in, int t, int c) {
    return rg_gelu_tanh(rg_in(in.fused, in.dtype, in.parts, in.part_stride, (size_t)t * in.row_stride + in.y_off + c) + in.y_bias[c]);
}

// a thread a channel: grid (ceil(W / 128), requests)
template <typename TO, bool MADE>
__global__ void __launch_bounds__(128)
rglru_walk_kernel(RgInput in, RgGates g, RgPairs src, const int* __restrict__ req_q_len, float* __restrict__ state, TO* __restrict__ out) {
    pdl_begin();
    const int r = blockIdx.y, len = req_q_len[r], slot = in.req_slot[r], c = blockIdx.x * 128 + threadIdx.x;
    if (len <= 0 || slot < 0 || c >= in.W) return;
    const int t0 = in.req_q_start[r];
    float S = state[(size_t)slot * in.W + c];
    for (int k0 = 0; k0 < len; k0 += 8) {
        float2 p[8];
        float y[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) p[u] = k0 + u < len ? rg_pair_at<MADE>(src, g, in.W, t0 + k0 + u, c) : make_float2(0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 8; ++u) y[u] = k0 + u < len ? rg_y(in, t0 + k0 + u, c) : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (k0 + u < len) {
                S = rg_advance(S, p[u]);
                out[(size_t)(t0 + k0 + u) * in.W + c] = from_f32<TO>(S * y[u]);
            }
    }
    state[(size_t)slot * in.W + c] = S;
    rg_keep_inputs(in, t0, len, slot, in.positions[t0], c);
}

// runs side by side: grid (ceil(W / 8), requests), 256 threads = 32 runs of 4 tokens by 8 channels; a warp has four runs
constexpr int RG_RUNS = 32, RG_RUN = 4, RG_COLS = 8, RG_WARPS = RG_RUNS * RG_COLS / 32;
// what a run's tokens bring, as it comes from memory
template <bool MADE> struct RgRaw;
template <> struct RgRaw<true> {
    float2 p[RG_RUN];
    __device__ __forceinline__ void load(const RgPairs& src, int W, int t0, int k0, int len, int c) {
#pragma unroll
        for (int u = 0; u < RG_RUN; ++u) p[u] = src.ab[(size_t)(t0 + min(k0 + u, len - 1)) * W + c];
    }
    __device__ __forceinline__ float2 pair(const RgGates&, int, int u) const { return p[u]; }
};
template <> struct RgRaw<false> {
    float zr[RG_RUN], zi[RG_RUN];
    bf16 hi[RG_RUN], lo[RG_RUN];
    __device__ __forceinline__ void load(const RgPairs& src, int, int t0, int k0, int len, int c) {
        const size_t base = (size_t)(c / src.s) * src.n * 2 * src.s + c % src.s;
#pragma unroll
        for (int u = 0; u < RG_RUN; ++u) {
            const size_t at = base + (size_t)(t0 + min(k0 + u, len - 1)) * 2 * src.s;
            zr[u] = src.z[at]; zi[u] = src.z[at + src.s];
            hi[u] = src.uv[at]; lo[u] = src.uv[at + src.s];
        }
    }
    __device__ __forceinline__ float2 pair(const RgGates& g, int c, int u) const {
        return rg_pair(g, c, zr[u], zi[u], __bfloat162float(hi[u]) + __bfloat162float(lo[u]));
    }
};
// two stretches of the recurrence one behind the other, each as (decay product - 1, end state from zero)
__device__ __forceinline__ float2 rg_join(float2 first, float2 second) {
    return make_float2(first.x + fmaf(second.x, first.x, second.x), rg_advance(first.y, second));
}
template <typename TO, bool MADE>
__global__ void __launch_bounds__(RG_RUNS * RG_COLS, 3)
rglru_runs_kernel(RgInput in, RgGates g, RgPairs src, const int* __restrict__ req_q_len, float* __restrict__ state, TO* __restrict__ out) {
    __shared__ float2 local[2][RG_WARPS][RG_COLS];       // a warp's four runs joined
    pdl_begin();
    const int r = blockIdx.y, len = req_q_len[r], slot = in.req_slot[r];
    if (len <= 0 || slot < 0) return;
    const int run = threadIdx.x / RG_COLS, col = threadIdx.x % RG_COLS, c = blockIdx.x * RG_COLS + col;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool live = c < in.W;
    const int cc = live ? c : in.W - 1;
    const int t0 = in.req_q_start[r];
    float carry = state[(size_t)slot * in.W + cc];      // the state in front of the tile
    const float y_bias = in.y_bias[cc];
    constexpr int TILE = RG_RUNS * RG_RUN;
    const int tiles = (len + TILE - 1) / TILE;
    RgRaw<MADE> raw;
    float y_raw[RG_RUN];
    auto load = [&](int tile) {
        const int k0 = tile * TILE + run * RG_RUN;
        raw.load(src, in.W, t0, k0, len, cc);
#pragma unroll
        for (int u = 0; u < RG_RUN; ++u)
            y_raw[u] = rg_in(in.fused, in.dtype, in.parts, in.part_stride, (size_t)(t0 + min(k0 + u, len - 1)) * in.row_stride + in.y_off + cc);
    };
    load(0);
    for (int tile = 0; tile < tiles; ++tile) {
        const int k0 = tile * TILE + run * RG_RUN;
        float2 p[RG_RUN];
        float y[RG_RUN];
#pragma unroll
        for (int u = 0; u < RG_RUN; ++u) {
            p[u] = raw.pair(g, cc, u);
            if (k0 + u >= len) p[u] = make_float2(0.f, 0.f);
            y[u] = y_raw[u];
        }
        if (tile + 1 < tiles) load(tile + 1);           // on its way while this tile is walked
        float2 mine = p[0];
#pragma unroll
        for (int u = 1; u < RG_RUN; ++u) mine = rg_join(mine, p[u]);
        // the runs of the warp that lie before this one, and the warp's four together
        float2 upto = mine;
#pragma unroll
        for (int o = RG_COLS; o < 32; o <<= 1) {
            const float2 before = make_float2(__shfl_up_sync(0xffffffffu, upto.x, o), __shfl_up_sync(0xffffffffu, upto.y, o));
            if (lane >= o) upto = rg_join(before, upto);
        }
        if (lane >= 32 - RG_COLS) local[tile & 1][warp][col] = upto;
        __syncthreads();                                // (the buffer of the tile before is read to its end by the time this one is full)
        float S = carry, end = carry;
#pragma unroll
        for (int w = 0; w < RG_WARPS; ++w) {
            if (w == warp) S = end;
            end = rg_advance(end, local[tile & 1][w][col]);
        }
        carry = end;
        const float2 before = make_float2(__shfl_up_sync(0xffffffffu, upto.x, RG_COLS), __shfl_up_sync(0xffffffffu, upto.y, RG_COLS));
        if (lane >= RG_COLS) S = rg_advance(S, before);
#pragma unroll
        for (int u = 0; u < RG_RUN; ++u) {
            S = rg_advance(S, p[u]);
            if (k0 + u < len && live) out[(size_t)(t0 + k0 + u) * in.W + c] = from_f32<TO>(S * rg_gelu_tanh(y[u] + y_bias));
        }
    }
    if (run == 0 && live) {
        state[(size_t)slot * in.W + c] = carry;
        rg_keep_inputs(in, t0, len, slot, in.positions[t0], c);
    }
}

// ---------------------------------------------------------------------------------------------------
// one token a request: grid (blocks x tiles of 32 channels, tiles of 16 tokens), 256 threads.  The block's channels of the tokens go
// to shared memory (convolution, high and low pieces); the warps share the block's channels among them (steps of 16), each
// runs the 64 rows of both maps against the tokens, and the sums meet in shared memory; then a thread a (token, channel).
// ---------------------------------------------------------------------------------------------------
constexpr int RS_TOK = 16, RS_COLS = 32, RS_MAX_S = 1024;
__host__ __device__ inline size_t rg_step_smem(int s) {
    const int pitch = ((s + 15) & ~15) + 8;
    return (size_t)2 * RS_TOK * pitch * 2 + (size_t)8 * 2 * RS_COLS * (RS_TOK + 1) * 4 + (size_t)RS_TOK * RS_COLS * 4;
}

template <typename TO>
__global__ void __launch_bounds__(256)
rglru_step_kernel(RgInput in, RgGates g, int n, const int* __restrict__ req_q_len, float* __restrict__ state, TO* __restrict__ out) {
    extern __shared__ __align__(16) unsigned char rg_smem[];
    const int sp = (g.s + 15) & ~15, pitch = sp + 8;
    bf16* hi = reinterpret_cast<bf16*>(rg_smem);                        // [16][pitch]
    bf16* lo = hi + RS_TOK * pitch;
    float* red = reinterpret_cast<float*>(lo + RS_TOK * pitch);         // [8 warps][64 rows][16 + 1 tokens]
    float* us = red + 8 * 2 * RS_COLS * (RS_TOK + 1);                   // [16][32] the tile's own channels
    pdl_launch_dependents();
    const int tiles = (g.s + RS_COLS - 1) / RS_COLS, b = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * RS_COLS, t0 = blockIdx.y * RS_TOK;
    const int base = b * g.s, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int steps = sp / 16;
    // rows of the maps as the left operand: m tile m of four (R's first and second 16 channels, then I's)
    auto load_a = [&](int ks, uint32_t (&a)[4][4]) {
#pragma unroll
        for (int m = 0; m < 4; ++m) {
            const bf16* w = reinterpret_cast<const bf16*>(m < 2 ? g.ra : g.ri);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int col = col0 + (m & 1) * 16 + (lane >> 2) + (q & 1) * 8, k = ks * 16 + (lane & 3) * 2 + (q >> 1) * 8;
                a[m][q] = (col < g.s && k < g.s) ? *reinterpret_cast<const uint32_t*>(w + b * g.block + (size_t)col * g.pitch + k) : 0u;
            }
        }
    };
    uint32_t a0[4][4], a1[4][4];
    if (warp < steps) load_a(warp, a0);                                 // (weights: asked for while the product before still runs)
    if (warp + 8 < steps) load_a(warp + 8, a1);
    pdl_wait();
    for (int idx = threadIdx.x; idx < RS_TOK * (sp / 8); idx += 256) {
        const int tt = idx / (sp / 8), k = (idx % (sp / 8)) * 8, t = t0 + tt;
        float u[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] = 0.f;
        if (t < n && k < g.s) {
            const int r = in.token_req[t];
            rg_conv8(in, t, t - in.req_q_start[r], max(in.req_slot[r], 0), in.positions[t], base + k, u);
        }
        uint4 h, l;
        rg_split2(u[0], u[1], h.x, l.x); rg_split2(u[2], u[3], h.y, l.y);
        rg_split2(u[4], u[5], h.z, l.z); rg_split2(u[6], u[7], h.w, l.w);
        *reinterpret_cast<uint4*>(hi + tt * pitch + k) = h;
        *reinterpret_cast<uint4*>(lo + tt * pitch + k) = l;
        if (k >= col0 && k < col0 + RS_COLS) {
#pragma unroll
            for (int e = 0; e < 8; ++e) us[tt * RS_COLS + k - col0 + e] = u[e];
        }
    }
    __syncthreads();
    float acc[4][2][4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
    auto multiply = [&](int ks, const uint32_t (&a)[4][4]) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int at = (j * 8 + (lane >> 2)) * pitch + ks * 16 + (lane & 3) * 2;
            const uint32_t h0 = *reinterpret_cast<const uint32_t*>(hi + at), h1 = *reinterpret_cast<const uint32_t*>(hi + at + 8);
            const uint32_t l0 = *reinterpret_cast<const uint32_t*>(lo + at), l1 = *reinterpret_cast<const uint32_t*>(lo + at + 8);
#pragma unroll
            for (int m = 0; m < 4; ++m) { rg_mma(acc[m][j], a[m], l0, l1); rg_mma(acc[m][j], a[m], h0, h1); }
        }
    };
    for (int ks = warp; ks < steps; ks += 16) {
        multiply(ks, a0);
        if (ks + 16 < steps) load_a(ks + 16, a0);
        if (ks + 8 < steps) {
            multiply(ks + 8, a1);
            if (ks + 24 < steps) load_a(ks + 24, a1);
        }
    }
    float* mine = red + (size_t)warp * 2 * RS_COLS * (RS_TOK + 1);
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int q = 0; q < 4; ++q)
                mine[(m * 16 + (lane >> 2) + (q >> 1) * 8) * (RS_TOK + 1) + j * 8 + (lane & 3) * 2 + (q & 1)] = acc[m][j][q];
    __syncthreads();
    for (int idx = threadIdx.x; idx < RS_TOK * RS_COLS; idx += 256) {
        const int tt = idx / RS_COLS, cc = idx % RS_COLS, t = t0 + tt, c = base + col0 + cc;
        if (t >= n || col0 + cc >= g.s) continue;
        const int r = in.token_req[t], slot = in.req_slot[r];
        if (req_q_len[r] <= 0 || slot < 0) continue;
        float zr = 0.f, zi = 0.f;
        for (int w = 0; w < 8; ++w) {
            zr += red[((size_t)w * 2 * RS_COLS + cc) * (RS_TOK + 1) + tt];
            zi += red[((size_t)w * 2 * RS_COLS + RS_COLS + cc) * (RS_TOK + 1) + tt];
        }
        const float2 p = rg_pair(g, c, zr, zi, us[tt * RS_COLS + cc]);
        const float S = rg_advance(state[(size_t)slot * in.W + c], p);
        state[(size_t)slot * in.W + c] = S;
        out[(size_t)t * in.W + c] = from_f32<TO>(S * rg_y(in, t, c));
        in.ring[((size_t)slot * in.T + in.positions[t] % in.T) * in.W + c] = rg_x(in, t, 0, slot, in.positions[t], 0, c);
    }
}

static int rg_check(const RgInput& in) {
    if (in.W <= 0 || in.T < 1 || in.parts < 1 || in.row_stride <= 0) return WLLM_BAD_SIZE;
    if ((in.dtype != WLLM_BF16 && in.dtype != WLLM_F32) || (in.parts > 1 && in.dtype != WLLM_F32)) return WLLM_BAD_DTYPE;
    if (!in.fused || !in.x_bias || !in.y_bias || !in.taps || !in.conv_bias || !in.positions || !in.token_req || !in.req_q_start ||
        !in.req_slot || !in.ring)
        return WLLM_BAD_SIZE;
    return WLLM_OK;
}
// rows, vectors and maps whose eight neighbouring elements may be read with 16-byte loads
static bool rg_wide(const RgInput& in, const RgGates& g) {
    return g.w_dtype == WLLM_BF16 && g.s % 8 == 0 && g.pitch % 8 == 0 && g.block % 8 == 0 && in.W % 8 == 0 && in.x_off % 8 == 0 && in.row_stride % 8 == 0 && in.part_stride % 4 == 0 &&
           !(((uintptr_t)in.fused | (uintptr_t)in.x_bias | (uintptr_t)in.taps | (uintptr_t)in.conv_bias | (uintptr_t)in.ring | (uintptr_t)g.ra |
              (uintptr_t)g.ri) & 15);
}

#define RG_INPUT_ARGS const void* fused, int in_dtype, int row_stride, int parts, long long part_stride, int y_off, int x_off, \
    const float* x_bias, const float* y_bias, const float* taps, const float* conv_bias, int T, int W, const int* positions, \
    const int* token_req, const int* req_q_start, const int* req_slot, float* ring
#define RG_INPUT RgInput{fused, in_dtype, row_stride, parts, (size_t)part_stride, y_off, x_off, x_bias, y_bias, taps, conv_bias, T, W, \
    positions, token_req, req_q_start, req_slot, ring}
#define RG_GATE_ARGS const void* ra, const void* ri, int w_dtype, int w_pitch, long long w_block, const float* ra_bias, const float* ri_bias, \
    const float* rate, int B
#define RG_GATES RgGates{ra, ri, w_dtype, w_pitch, (size_t)w_block, ra_bias, ri_bias, rate, B, B > 0 ? W / B : 0}

static int rg_gates_ok(const RgGates& g, int W) {
    if (g.B < 1 || W % g.B != 0 || !g.ra || !g.ri || !g.ra_bias || !g.ri_bias || !g.rate || g.pitch < g.s) return WLLM_BAD_SIZE;
    return g.w_dtype == WLLM_BF16 || g.w_dtype == WLLM_F32 ? WLLM_OK : WLLM_BAD_DTYPE;
}

// ab [n, W, 2]
WLLM_API int wllm_rglru_gates(RG_INPUT_ARGS, RG_GATE_ARGS, int n, float* ab, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    const RgInput in = RG_INPUT;
    int st = rg_check(in);
    if (st != WLLM_OK) return st;
    const RgGates g = RG_GATES;
    st = rg_gates_ok(g, W);
    if (st != WLLM_OK) return st;
    if (rg_wide(in, g) && ((uintptr_t)ab & 15) == 0) {
        static bool raised = false;
        if (!raised) {
            const cudaError_t e = cudaFuncSetAttribute(rglru_gates_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(RgSmem));
            if (e != cudaSuccess) return 1000 + (int)e;
            raised = true;
        }
        const dim3 grid(B * ((g.s + RG_TN - 1) / RG_TN), (n + RG_TM - 1) / RG_TM);
        if (grid.y > 65535) return WLLM_BAD_SIZE;
        return wllm_launch(rglru_gates_mma_kernel, grid, 256, sizeof(RgSmem), stream, in, g, n, (float2*)ab);
    }
    const dim3 grid(B * ((g.s + 31) / 32), (n + 31) / 32);
    if (grid.y > 65535) return WLLM_BAD_SIZE;
    return wllm_launch(rglru_gates_plain_kernel, grid, 256, 0, stream, in, g, n, (float2*)ab);
}

// uv [B][n][2 W / B] (see above); tiles (null: none): 1 + 3 * B * ceil(n / tile_rows) ints.  W / B in steps of 8, aligned rows.
WLLM_API int wllm_rglru_conv(RG_INPUT_ARGS, int B, int n, void* uv, int* tiles, int tile_rows, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    const RgInput in = RG_INPUT;
    const int st = rg_check(in);
    if (st != WLLM_OK) return st;
    if (B < 1 || W % B != 0 || (W / B) % 8 != 0 || in.x_off % 8 != 0 || in.row_stride % 8 != 0 || in.part_stride % 4 != 0 || (tiles && tile_rows < 1))
        return WLLM_BAD_SIZE;
    if (((uintptr_t)fused | (uintptr_t)x_bias | (uintptr_t)taps | (uintptr_t)conv_bias | (uintptr_t)ring | (uintptr_t)uv) & 15) return WLLM_BAD_ALIGN;
    return wllm_launch(rglru_conv_kernel, dim3((n + 3) / 4, (W + 511) / 512), 256, 0, stream, in, n, B, W / B, (bf16*)uv, tiles, tile_rows);
}

// ab [n, W, 2], or (ab null) z [B][n][2 W / B] and uv of the same shape: n tokens.  long_portions: the step holds portions long enough
// for runs side by side (else every request is walked token by token)
WLLM_API int wllm_rglru_scan(RG_INPUT_ARGS, RG_GATE_ARGS, int n, const float* ab, const float* z, const void* uv, const int* req_q_len,
                             int requests, float* state, void* out, int out_dtype, int long_portions, cudaStream_t stream) {
    if (requests <= 0) return WLLM_OK;
    const RgInput in = RG_INPUT;
    int st = rg_check(in);
    if (st != WLLM_OK) return st;
    const RgGates g = RG_GATES;
    st = rg_gates_ok(g, W);
    if (st != WLLM_OK) return st;
    if (requests > 65535 || (!ab && (!z || !uv)) || !state || !out) return WLLM_BAD_SIZE;
    const RgPairs src{(const float2*)ab, z, (const bf16*)uv, n, g.s};
#define GO2(TO, M) (long_portions \
        ? wllm_launch(rglru_runs_kernel<TO, M>, dim3((W + RG_COLS - 1) / RG_COLS, requests), RG_RUNS * RG_COLS, 0, stream, in, g, src, req_q_len, state, (TO*)out) \
        : wllm_launch(rglru_walk_kernel<TO, M>, dim3((W + 127) / 128, requests), 128, 0, stream, in, g, src, req_q_len, state, (TO*)out))
#define GO(TO) (ab ? GO2(TO, true) : GO2(TO, false))
    if (out_dtype == WLLM_BF16) return GO(bf16);
    if (out_dtype == WLLM_F32) return GO(float);
#undef GO
#undef GO2
    return WLLM_BAD_DTYPE;
}

// No request of the step may bring more than one token.  Blocks of up to 1,024 channels in steps of 8, bfloat16 maps.
WLLM_API int wllm_rglru_step(RG_INPUT_ARGS, RG_GATE_ARGS, int n, const int* req_q_len, float* state, void* out, int out_dtype,
                             cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    const RgInput in = RG_INPUT;
    int st = rg_check(in);
    if (st != WLLM_OK) return st;
    const RgGates g = RG_GATES;
    st = rg_gates_ok(g, W);
    if (st != WLLM_OK) return st;
    if (!rg_wide(in, g) || g.s > RS_MAX_S) return WLLM_BAD_SIZE;
    if (out_dtype != WLLM_BF16) return WLLM_BAD_DTYPE;
    static bool raised = false;
    if (!raised) {
        const cudaError_t e = cudaFuncSetAttribute(rglru_step_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)rg_step_smem(RS_MAX_S));
        if (e != cudaSuccess) return 1000 + (int)e;
        raised = true;
    }
    const dim3 grid(B * ((g.s + RS_COLS - 1) / RS_COLS), (n + RS_TOK - 1) / RS_TOK);
    if (grid.y > 65535) return WLLM_BAD_SIZE;
    return wllm_launch(rglru_step_kernel<bf16>, grid, 256, rg_step_smem(g.s), stream, in, g, n, req_q_len, state, (bf16*)out);
}
