// Blends of a token's row with the row of the token before it, and the products that read them.
//
//     x_s[t] = h[t] + (h[t - 1] - h[t]) * mu_s            one weight per channel and stream s; the row before the first is zero
//
// h[t - 1] is the step's own row when the request's portion reaches back that far, else the row its slot kept: two rows a slot,
// the row of position p in row p mod 2, so a step of single tokens reads one and writes the other.
//
//   wllm_token_blend      the S blends of every token, [S, n, H], rounded once (the operands of the products), the slots' rows, and,
//                         for the grouped product that takes several streams at once, its table of row tiles.  A thread has eight
//                         channels (or one) of a run of tokens.
//   wllm_blended_product  few tokens, one a request (decoding), bfloat16: the products themselves, each reading its own blend.  The
//                         matrices lie one below the other, [N, H], in segments that name their stream (or none: h itself);
//                         out [n, N] 32-bit.  A CTA has some rows of one segment, so many that all CTAs run at once: it blends the
//                         tokens' rows into shared memory once and walks its rows sixteen at a time; its eight warps share K (32
//                         columns at a time, every lane 16 contiguous bytes of a row, the first asked for while the kernel before
//                         still runs, the next rows' while these are multiplied), and their sums meet in shared memory in warp order.
#include "common.cuh"

constexpr int TB_MAX_STREAMS = 8, TB_TOKENS = 8;

template <typename T, int VEC> struct TbRow;
template <> struct TbRow<bf16, 8> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[8]) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h2[e]); v[2 * e] = f.x; v[2 * e + 1] = f.y; }
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[8]) {
        uint4 raw;
        __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};
template <typename T> struct TbRow<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32(*p); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};

// grid (tiles of TB_TOKENS tokens, tiles of 128 * VEC channels), 128 threads
template <typename T, int VEC, int S>
__global__ void __launch_bounds__(128)
token_blend_kernel(const T* __restrict__ h, int n, int H, const float* __restrict__ mu, const int* __restrict__ positions,
                   const int* __restrict__ token_req, const int* __restrict__ req_q_start, const int* __restrict__ req_q_len,
                   const int* __restrict__ req_slot, T* __restrict__ kept, T* __restrict__ out, int* __restrict__ tiles, int groups,
                   int tile_rows) {
    pdl_begin();
    if (tiles != nullptr && blockIdx.x == 0 && blockIdx.y == 0) {       // (group, first row, rows) of every row tile of n rows a group
        const int per = (n + tile_rows - 1) / tile_rows;
        for (int i = threadIdx.x; i < groups * per; i += blockDim.x) {
            const int g = i / per, k = i % per;
            tiles[1 + 3 * i] = g;
            tiles[2 + 3 * i] = g * n + k * tile_rows;
            tiles[3 + 3 * i] = min(tile_rows, n - k * tile_rows);
        }
        if (threadIdx.x == 0) tiles[0] = groups * per;
    }
    const int c = (blockIdx.y * 128 + threadIdx.x) * VEC;
    if (c >= H) return;
    float m[S][VEC];
#pragma unroll
    for (int s = 0; s < S; ++s)
#pragma unroll
        for (int e = 0; e < VEC; ++e) m[s][e] = mu[(size_t)s * H + c + e];
    const int t_lo = blockIdx.x * TB_TOKENS, t_hi = min(n, t_lo + TB_TOKENS);
    float before[VEC];
    bool have = false;                     // `before` holds the row of the token in front of t
    for (int t = t_lo; t < t_hi; ++t) {
        const int r = token_req[t], q0 = req_q_start[r], len = req_q_len[r], slot = req_slot[r], pos = positions[t];
        if (t > q0) {
            if (!have) TbRow<T, VEC>::load(h + (size_t)(t - 1) * H + c, before);
        } else if (pos > 0 && len > 0 && slot >= 0) {
            TbRow<T, VEC>::load(kept + ((size_t)slot * 2 + ((pos - 1) & 1)) * H + c, before);
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) before[e] = 0.f;
        }
        float x[VEC], y[VEC];
        TbRow<T, VEC>::load(h + (size_t)t * H + c, x);
#pragma unroll
        for (int s = 0; s < S; ++s) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] = fmaf(before[e] - x[e], m[s][e], x[e]);
            TbRow<T, VEC>::store(out + ((size_t)s * n + t) * H + c, y);
        }
        if (t == q0 && len > 0 && slot >= 0) {
            // the thread that has read the kept row of these channels (no other reads it) leaves the portion's last row
            float last[VEC];
            TbRow<T, VEC>::load(h + (size_t)(q0 + len - 1) * H + c, last);
            TbRow<T, VEC>::store(kept + ((size_t)slot * 2 + ((pos + len - 1) & 1)) * H + c, last);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) before[e] = x[e];
        have = t + 1 < t_hi && token_req[t + 1] == r;
    }
}

// tiles (null: none): 1 + 3 * groups * ceil(n / tile_rows) ints; mu [S][H]; kept [slots][2][H] and out [S][n][H] of h's element type
WLLM_API int wllm_token_blend(const void* h, int dtype, int n, int H, const float* mu, int S, const int* positions, const int* token_req,
                              const int* req_q_start, const int* req_q_len, const int* req_slot, void* kept, void* out, int* tiles,
                              int groups, int tile_rows, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (H <= 0 || S < 1 || S > TB_MAX_STREAMS || (tiles != nullptr && (groups < 1 || tile_rows < 1))) return WLLM_BAD_SIZE;
    const bool vec = dtype == WLLM_BF16 && H % 8 == 0 && !(((uintptr_t)h | (uintptr_t)kept | (uintptr_t)out) & 15);
    const int per = vec ? 8 : 1;
    const dim3 grid((n + TB_TOKENS - 1) / TB_TOKENS, (H + 128 * per - 1) / (128 * per));
#define GO(T, V, SS) wllm_launch(token_blend_kernel<T, V, SS>, grid, 128, 0, stream, (const T*)h, n, H, mu, positions, token_req, req_q_start, \
        req_q_len, req_slot, (T*)kept, (T*)out, tiles, groups, tile_rows)
#define PICK(SS) (vec ? GO(bf16, 8, SS) : dtype == WLLM_BF16 ? GO(bf16, 1, SS) : GO(float, 1, SS))
    if (dtype != WLLM_BF16 && dtype != WLLM_F32) return WLLM_BAD_DTYPE;
    switch (S) {
        case 1: return PICK(1); case 2: return PICK(2); case 3: return PICK(3); case 4: return PICK(4);
        case 5: return PICK(5); case 6: return PICK(6); case 7: return PICK(7); case 8: return PICK(8);
    }
#undef PICK
#undef GO
    return WLLM_BAD_SIZE;
}

// ---------------------------------------------------------------------------------------------------
// products of blends, few tokens
// ---------------------------------------------------------------------------------------------------
struct BlendSegments {
    int count;
    int row0[TB_MAX_STREAMS + 1];        // first row of a segment; row0[count] = N
    int stream[TB_MAX_STREAMS + 1];      // the stream it reads, -1: h itself
    int tile0[TB_MAX_STREAMS + 1];       // first CTA
};
constexpr int BP_ROWS = 16, BP_WARPS = 8, BP_CTAS = 2 * 148;

__device__ __forceinline__ void bp_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 bp_stream(const bf16* p) {              // weights: read once a step
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// NT: tiles of eight tokens; DEPTH: runs of 32 columns a warp has on their way.  KC: columns of the tokens' blends that lie in shared memory
// at a time (all of them, or a multiple of 256 * DEPTH); subs: groups of sixteen rows of a CTA (1 when the blends do not fit at once).
template <int NT, int DEPTH>
__global__ void __launch_bounds__(BP_WARPS * 32, 2)
blended_product_kernel(const bf16* __restrict__ h, int n, int H, const float* __restrict__ mu, const bf16* __restrict__ w, BlendSegments seg,
                       const int* __restrict__ positions, const int* __restrict__ token_req, const int* __restrict__ req_q_len,
                       const int* __restrict__ req_slot, bf16* __restrict__ kept, float* __restrict__ out, int N, int KC, int subs) {
    extern __shared__ __align__(16) unsigned char bp_smem[];
    constexpr int RP = 8 * NT + 1;
    bf16* xs = reinterpret_cast<bf16*>(bp_smem);                                      // [8 NT][KC + 8]
    float* red = reinterpret_cast<float*>(bp_smem + (size_t)8 * NT * (KC + 8) * 2);   // [2][8 warps][16 rows][8 NT + 1]
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pitch = KC + 8;
    int sg = 0;
    while (sg + 1 < seg.count && (int)blockIdx.x >= seg.tile0[sg + 1]) ++sg;
    const int row0 = seg.row0[sg] + ((int)blockIdx.x - seg.tile0[sg]) * BP_ROWS * subs, row_end = min(seg.row0[sg + 1], row0 + BP_ROWS * subs);
    const int stream = seg.stream[sg];
    // this lane's rows of a group (lane / 4 and that + 8) and its 16-byte piece of a run of 32 columns; a warp's runs are warp, warp + 8, ..,
    // padded to whole rounds of DEPTH
    const int steps = (H + 31) / 32, mine = steps > warp ? (steps - warp + BP_WARPS - 1) / BP_WARPS : 0;
    const int rounds = ((steps + BP_WARPS - 1) / BP_WARPS + DEPTH - 1) / DEPTH;
    uint4 a[DEPTH][2];
    auto fetch = [&](int sub, int q, uint4 (&to)[2]) {
        const int k = (warp + q * BP_WARPS) * 32 + (lane & 3) * 8;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int row = row0 + sub * BP_ROWS + (lane >> 2) + 8 * j;
            to[j] = (q < mine && row < row_end && k < H) ? bp_stream(w + (size_t)row * H + k) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
#pragma unroll
    for (int q = 0; q < DEPTH; ++q) fetch(0, q, a[q]);
    pdl_wait();
    auto blend = [&](int k0) {
        for (int idx = threadIdx.x; idx < 8 * NT * (KC / 8); idx += blockDim.x) {
            const int tt = idx / (KC / 8), c = k0 + (idx % (KC / 8)) * 8;
            uint4 packed = make_uint4(0u, 0u, 0u, 0u);
            if (tt < n && c < H) {
                packed = *reinterpret_cast<const uint4*>(h + (size_t)tt * H + c);
                const int r = token_req[tt], slot = req_slot[r], pos = positions[tt];
                const bool live = req_q_len[r] > 0 && slot >= 0;
                if (blockIdx.x == 0 && live) *reinterpret_cast<uint4*>(kept + ((size_t)slot * 2 + (pos & 1)) * H + c) = packed;
                if (stream >= 0) {
                    float x[8], b[8], y[8];
                    TbRow<bf16, 8>::load(reinterpret_cast<const bf16*>(&packed), x);
#pragma unroll
                    for (int e = 0; e < 8; ++e) b[e] = 0.f;
                    if (live && pos > 0) TbRow<bf16, 8>::load(kept + ((size_t)slot * 2 + ((pos - 1) & 1)) * H + c, b);
                    const float4 m0 = *reinterpret_cast<const float4*>(mu + (size_t)stream * H + c), m1 = *reinterpret_cast<const float4*>(mu + (size_t)stream * H + c + 4);
                    const float m[8] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] = fmaf(b[e] - x[e], m[e], x[e]);
                    TbRow<bf16, 8>::store(reinterpret_cast<bf16*>(&packed), y);
                }
            }
            *reinterpret_cast<uint4*>(xs + tt * pitch + (c - k0)) = packed;
        }
    };
    const int per_chunk = KC / (32 * BP_WARPS);                 // runs a warp has in a chunk
    const bool whole = KC >= H;
    if (whole) { blend(0); __syncthreads(); }
    for (int sub = 0; sub < subs && row0 + sub * BP_ROWS < row_end; ++sub) {
        float acc[NT][4];
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        int k0 = 0, base = 0;                                   // first column and first run of the chunk that lies in shared memory
        if (!whole) { blend(0); __syncthreads(); }
        for (int round = 0; round < rounds; ++round) {
            if (!whole && round * DEPTH >= base + per_chunk) {  // (a chunk holds whole rounds)
                __syncthreads();
                k0 += KC; base += per_chunk;
                blend(k0);
                __syncthreads();
            }
#pragma unroll
            for (int d = 0; d < DEPTH; ++d) {
                const int q = round * DEPTH + d;
                if (q < mine) {
                    const int col = (warp + q * BP_WARPS) * 32 - k0 + (lane & 3) * 8;
#pragma unroll
                    for (int j = 0; j < NT; ++j) {
                        const uint4 b = *reinterpret_cast<const uint4*>(xs + (j * 8 + (lane >> 2)) * pitch + col);
                        // a lane's eight columns of a run are the columns of two steps of 16: which of them stands where does
                        // not matter to the sum, as long as both operands agree
                        bp_mma(acc[j], a[d][0].x, a[d][1].x, a[d][0].y, a[d][1].y, b.x, b.y);
                        bp_mma(acc[j], a[d][0].z, a[d][1].z, a[d][0].w, a[d][1].w, b.z, b.w);
                    }
                }
                if (round + 1 < rounds) fetch(sub, q + DEPTH, a[d]);
                else if (sub + 1 < subs) fetch(sub + 1, d, a[d]);
            }
        }
        // the warps' sums meet in one of two places: who writes the next ones does not meet who still reads these
        float* meet = red + (size_t)(sub & 1) * BP_WARPS * BP_ROWS * RP;
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int q = 0; q < 4; ++q)
                meet[((size_t)warp * BP_ROWS + (lane >> 2) + (q >> 1) * 8) * RP + j * 8 + (lane & 3) * 2 + (q & 1)] = acc[j][q];
        __syncthreads();
        for (int idx = threadIdx.x; idx < n * BP_ROWS; idx += blockDim.x) {
            const int tt = idx / BP_ROWS, row = idx % BP_ROWS, at = row0 + sub * BP_ROWS + row;
            if (at >= row_end) continue;
            float v = 0.f;
#pragma unroll
            for (int k = 0; k < BP_WARPS; ++k) v += meet[((size_t)k * BP_ROWS + row) * RP + tt];
            out[(size_t)tt * N + at] = v;
        }
    }
}

// rows[i]: matrix rows of segment i, streams[i]: the blend it reads (-1: h itself); `count` segments, at most 9.  n up to 32, H in steps of 8,
// no request with more than one token.  out [n, sum of rows]
WLLM_API int wllm_blended_product(const void* h, int n, int H, const float* mu, const void* w, const int* rows, const int* streams, int count,
                                  const int* positions, const int* token_req, const int* req_q_len, const int* req_slot, void* kept,
                                  float* out, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (n > 32 || H <= 0 || H % 8 != 0 || count < 1 || count > TB_MAX_STREAMS) return WLLM_BAD_SIZE;
    if (((uintptr_t)h | (uintptr_t)w | (uintptr_t)kept | (uintptr_t)mu) & 15) return WLLM_BAD_ALIGN;
    BlendSegments seg = {};
    seg.count = count;
    const int nt = n <= 8 ? 1 : (n <= 16 ? 2 : 4), depth = nt == 4 ? 4 : 8;
    const int round = 32 * BP_WARPS * depth;
    // the blends in shared memory: whole rows of the tokens where they fit in some 66 KB, else as many columns as do, in whole rounds
    int kc = (H + 255) / 256 * 256;
    const int most = (33 * 1024 / (8 * nt) - 8) / round * round;
    if (kc > most) kc = most;
    int groups = 0;
    for (int i = 0; i < count; ++i) groups += (rows[i] + BP_ROWS - 1) / BP_ROWS;
    const int subs = kc < H ? 1 : (groups + BP_CTAS - 1) / BP_CTAS;
    int tiles = 0;
    for (int i = 0; i < count; ++i) {
        if (rows[i] < 1 || streams[i] < -1 || streams[i] >= TB_MAX_STREAMS) return WLLM_BAD_SIZE;
        seg.stream[i] = streams[i];
        seg.tile0[i] = tiles;
        seg.row0[i + 1] = seg.row0[i] + rows[i];
        tiles += (rows[i] + BP_ROWS * subs - 1) / (BP_ROWS * subs);
    }
    const int N = seg.row0[count];
    const size_t smem = (size_t)8 * nt * (kc + 8) * 2 + (size_t)2 * BP_WARPS * BP_ROWS * (8 * nt + 1) * 4;
#define GO(NT, D) do { \
        static bool raised = false; \
        if (!raised) { \
            const cudaError_t e = cudaFuncSetAttribute(blended_product_kernel<NT, D>, cudaFuncAttributeMaxDynamicSharedMemorySize, 110 * 1024); \
            if (e != cudaSuccess) return 1000 + (int)e; \
            raised = true; \
        } \
        return wllm_launch(blended_product_kernel<NT, D>, tiles, BP_WARPS * 32, smem, stream, (const bf16*)h, n, H, mu, (const bf16*)w, seg, positions, \
                           token_req, req_q_len, req_slot, (bf16*)kept, out, N, kc, subs); \
    } while (0)
    if (nt == 1) GO(1, 8);
    if (nt == 2) GO(2, 8);
    GO(4, 4);
#undef GO
}
