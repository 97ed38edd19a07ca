// A state space with a scalar decay per head and token (Mamba-2): a matrix state S [N, V] per (request, head), 32-bit,
//
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T,    y_t = S_t^T C_t + D_h x_t,    a_t = exp(-exp(A_log_h) dt_t)
//
// B and C are rows of N shared by the heads of a group, x the head's V values.  The recurrence itself is the decayed-state scan of
// linear_attention.cu (q = C, k = B, v = x, with a pair (a - 1, dt) per head and token); here is what stands in front of it
// and behind it.  All of it is 32-bit inside; inputs come from one fused projection row z | x | B | C | dt, possibly in split-K slabs.
//
//   wllm_ssd_prepare      the causal convolution of x | B | C along the sequence, channel by channel (`taps` taps, the last weighs the
//                         token itself, inputs in front of the sequence count as zero), its bias, SiLU: one 32-bit row a token; and
//                         dt = softplus(dt + dt_bias) with a - 1 = expm1(-exp(A_log) dt) (a head that forgets slowly has a close to
//                         one, and the rounding of a itself would grow with its memory).  In a step of single tokens it also
//                         shifts the slots' inputs: the thread that read a channel's writes them.
//   wllm_ssd_conv_update  the slots' last taps - 1 inputs after this step's tokens, for steps with portions.
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
template <int TT, int TAPS, bool MULTI>
__global__ void __launch_bounds__(256)
ssd_prepare_kernel(const void* __restrict__ fused, int in_dtype, int row_stride, int parts, size_t part_stride, int x_off, int dt_off,
                   int n, int C, int H, int any_taps, const void* __restrict__ conv, const void* __restrict__ conv_bias,
                   const void* __restrict__ a_log, const void* __restrict__ dt_bias, int w_dtype, const int* __restrict__ token_req,
                   const int* __restrict__ req_q_start, const int* __restrict__ req_q_len, const int* __restrict__ req_slot,
                   float* __restrict__ conv_state, float* __restrict__ out, float* __restrict__ pairs, int shift) {
    pdl_begin();
    const int t0 = blockIdx.x * TT, count = min(TT, n - t0);
    if (blockIdx.y == gridDim.y - 1) {
        for (int idx = threadIdx.x; idx < count * H; idx += blockDim.x) {
            const int t = t0 + idx / H, h = idx % H;
            const float z = ss_in<MULTI>(fused, in_dtype, parts, part_stride, (size_t)t * row_stride + dt_off + h) + ss_any(dt_bias, w_dtype, h);
            const float step = z > 20.f ? z : log1pf(expf(z));
            pairs[((size_t)t * H + h) * 2] = expm1f(-expf(ss_any(a_log, w_dtype, h)) * step);
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
        out[(size_t)t * C + ch] = ss_silu(acc);
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
            out[(size_t)t * C + ch] = ss_silu(acc);
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

// grid (tokens, groups): the part of the row in shared memory between its sum of squares (a block sum in a fixed order) and the scaling
template <typename TO, bool MULTI>
__global__ void ssd_gate_norm_kernel(const float* __restrict__ o, const float* __restrict__ x, size_t x_stride, const void* __restrict__ skip,
                                     const void* __restrict__ fused, int in_dtype, int row_stride, int parts, size_t part_stride, int z_off,
                                     const void* __restrict__ w, int w_dtype, float eps, TO* __restrict__ out, int inner, int V, int part) {
    extern __shared__ float ss_row[];
    __shared__ float scratch[32];
    pdl_begin();
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* orow = o + (size_t)t * inner + c0;
    const float* xrow = x + (size_t)t * x_stride + c0;
    const size_t zrow = (size_t)t * row_stride + z_off + c0;
    float ss = 0.f;
    for (int c = threadIdx.x; c < part; c += blockDim.x) {
        const float z = ss_in<MULTI>(fused, in_dtype, parts, part_stride, zrow + c);
        const float y = fmaf(ss_any(skip, w_dtype, (c0 + c) / V), xrow[c], orow[c]) * ss_silu(z);
        ss_row[c] = y;
        ss = fmaf(y, y, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    TO* dst = out + (size_t)t * inner + c0;
    for (int c = threadIdx.x; c < part; c += blockDim.x) dst[c] = from_f32<TO>((ss_row[c] * inv) * ss_any(w, w_dtype, c0 + c));
}

// The same for bfloat16 rows whose parts and heads come in steps of 4 elements: 16-byte loads of o and x, 8-byte loads of the gate and
// the gain, 8-byte stores.
__global__ void ssd_gate_norm_vec_kernel(const float* __restrict__ o, const float* __restrict__ x, size_t x_stride, const bf16* __restrict__ skip,
                                         const bf16* __restrict__ fused, int row_stride, int z_off, const bf16* __restrict__ w, float eps,
                                         bf16* __restrict__ out, int inner, int V, int part) {
    extern __shared__ float ss_row[];
    __shared__ float scratch[32];
    pdl_begin();
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* orow = o + (size_t)t * inner + c0;
    const float* xrow = x + (size_t)t * x_stride + c0;
    const bf16* zrow = fused + (size_t)t * row_stride + z_off + c0;
    float ss = 0.f;
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
        const float4 o4 = *reinterpret_cast<const float4*>(orow + c), x4 = *reinterpret_cast<const float4*>(xrow + c);
        const uint2 zr = *reinterpret_cast<const uint2*>(zrow + c);
        const float2 za = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zr.x));
        const float2 zb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zr.y));
        const float d = __bfloat162float(skip[(c0 + c) / V]);
        float4 y;
        y.x = fmaf(d, x4.x, o4.x) * ss_silu(za.x); y.y = fmaf(d, x4.y, o4.y) * ss_silu(za.y);
        y.z = fmaf(d, x4.z, o4.z) * ss_silu(zb.x); y.w = fmaf(d, x4.w, o4.w) * ss_silu(zb.y);
        *reinterpret_cast<float4*>(ss_row + c) = y;
        ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    bf16* dst = out + (size_t)t * inner + c0;
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
        const float4 y = *reinterpret_cast<const float4*>(ss_row + c);
        const uint2 wr = *reinterpret_cast<const uint2*>(w + c0 + c);
        const float2 wa = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&wr.x));
        const float2 wb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&wr.y));
        const __nv_bfloat162 a = __floats2bfloat162_rn((y.x * inv) * wa.x, (y.y * inv) * wa.y);
        const __nv_bfloat162 b = __floats2bfloat162_rn((y.z * inv) * wb.x, (y.w * inv) * wb.y);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&a);
        packed.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(dst + c) = packed;
    }
}

// fused [n, W] (or `parts` 32-bit slabs): x | B | C at x_off (C columns), dt at dt_off [H]; conv [C, taps], conv_bias [C] (may be null),
// a_log, dt_bias [H] of one element type; conv_state [slots, taps - 1, C]; out [n, C], pairs [n, H, 2] = (a - 1, dt), 32-bit.
// shift: every request of the step brings at most one token, and conv_state is brought up to date here.
WLLM_API int wllm_ssd_prepare(const void* fused, int in_dtype, int row_stride, int parts, long long part_stride, int x_off, int dt_off, int n,
                              int C, int H, int taps, const void* conv, const void* conv_bias, const void* a_log, const void* dt_bias,
                              int w_dtype, const int* token_req, const int* req_q_start, const int* req_q_len, const int* req_slot,
                              float* conv_state, float* out, float* pairs, int shift, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (C <= 0 || H <= 0 || taps < 1 || taps > SS_MAX_TAPS || parts < 1 || (taps > 1 && conv_state == nullptr)) return WLLM_BAD_SIZE;
    if ((in_dtype != WLLM_BF16 && in_dtype != WLLM_F32) || (w_dtype != WLLM_BF16 && w_dtype != WLLM_F32)) return WLLM_BAD_DTYPE;
    const int rows = (C + 255) / 256 + 1;
    if (rows > 65535) return WLLM_BAD_SIZE;
#define PREP(TT, TAPS, M) wllm_launch(ssd_prepare_kernel<TT, TAPS, M>, dim3((n + TT - 1) / TT, rows), 256, 0, stream, fused, in_dtype, row_stride, \
        parts, (size_t)part_stride, x_off, dt_off, n, C, H, taps, conv, conv_bias, a_log, dt_bias, w_dtype, token_req, req_q_start, req_q_len, \
        req_slot, conv_state, out, pairs, shift)
    if (parts == 1 && n >= 256 && !shift) {      // many tokens: a tile's inputs are loaded once
        if (taps == 2) return PREP(8, 2, false);
        if (taps == 3) return PREP(8, 3, false);
        if (taps == 4) return PREP(8, 4, false);
    }
    if (taps == 4) return parts > 1 ? PREP(1, 4, true) : PREP(1, 4, false);
    return parts > 1 ? PREP(1, 0, true) : PREP(1, 0, false);
#undef PREP
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

// o [n, inner], x [n, ..] with rows x_stride apart, 32-bit; skip [inner / V] and w [inner] of one element type; the gate z at z_off of fused
WLLM_API int wllm_ssd_gate_norm(const float* o, const float* x, long long x_stride, const void* skip, const void* fused, int in_dtype,
                                int row_stride, int parts, long long part_stride, int z_off, const void* w, int w_dtype, float eps, void* out,
                                int out_dtype, int n, int inner, int V, int groups, cudaStream_t stream) {
    if (n <= 0) return WLLM_OK;
    if (inner <= 0 || V <= 0 || inner % V != 0 || groups < 1 || groups > 65535 || inner % groups != 0 || parts < 1 || x_stride < inner)
        return WLLM_BAD_SIZE;
    if ((in_dtype != WLLM_BF16 && in_dtype != WLLM_F32) || (w_dtype != WLLM_BF16 && w_dtype != WLLM_F32)) return WLLM_BAD_DTYPE;
    const int part = inner / groups;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 192 * 1024) return WLLM_BAD_SIZE;
    static bool raised = false;
    if (!raised && smem > 48 * 1024) {
        cudaError_t e = cudaSuccess;
#define RAISE(K) if (e == cudaSuccess) e = cudaFuncSetAttribute(K, cudaFuncAttributeMaxDynamicSharedMemorySize, 192 * 1024)
        RAISE((ssd_gate_norm_kernel<bf16, true>)); RAISE((ssd_gate_norm_kernel<bf16, false>));
        RAISE((ssd_gate_norm_kernel<float, true>)); RAISE((ssd_gate_norm_kernel<float, false>));
        RAISE(ssd_gate_norm_vec_kernel);
#undef RAISE
        if (e != cudaSuccess) return 1000 + (int)e;
        raised = true;
    }
    const dim3 grid(n, groups);
    if (parts == 1 && in_dtype == WLLM_BF16 && w_dtype == WLLM_BF16 && out_dtype == WLLM_BF16 && part % 4 == 0 && V % 4 == 0 && x_stride % 4 == 0 &&
        row_stride % 4 == 0 && z_off % 4 == 0 && !(((uintptr_t)o | (uintptr_t)x) & 15) && !(((uintptr_t)fused | (uintptr_t)w | (uintptr_t)out) & 7)) {
        const int threads = part >= 2048 ? 256 : (part >= 512 ? 128 : 64);
        return wllm_launch(ssd_gate_norm_vec_kernel, grid, threads, smem, stream, o, x, (size_t)x_stride, (const bf16*)skip, (const bf16*)fused,
                           row_stride, z_off, (const bf16*)w, eps, (bf16*)out, inner, V, part);
    }
    const int threads = part >= 2048 ? 512 : (part >= 512 ? 256 : 128);
#define GATE(TO, M) wllm_launch(ssd_gate_norm_kernel<TO, M>, grid, threads, smem, stream, o, x, (size_t)x_stride, skip, fused, in_dtype, row_stride, \
        parts, (size_t)part_stride, z_off, w, w_dtype, eps, (TO*)out, inner, V, part)
    if (out_dtype == WLLM_BF16) return parts > 1 ? GATE(bf16, true) : GATE(bf16, false);
    if (out_dtype == WLLM_F32) return parts > 1 ? GATE(float, true) : GATE(float, false);
#undef GATE
    return WLLM_BAD_DTYPE;
}
