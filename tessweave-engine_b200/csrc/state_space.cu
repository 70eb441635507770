// The state-space recurrence of linear_recurrence.cu (TW_REC_SSD) for portions of a prompt, in chunks on the tensor cores.
//
// With a_t = -r dt_t (r the head's rate, dt_t the step size) and A_t = a_1 + ... + a_t inside a chunk of 64 tokens,
//
//   y_t   = e^(A_t) S^T c_t + sum over s <= t of e^(A_t - A_s) dt_s (c_t . b_s) x_s + u x_t       S: the state before the chunk
//   S_new = e^(A_64) S + sum over s of e^(A_64 - A_s) dt_s b_s x_s^T
//
// so a chunk is four matrix products (mma.sync m16n8k16, bf16 operands, fp32 sums): G = C B^T (the part at and below the
// diagonal), Y = C S, Y += M X with M = G times the decays and step sizes, and S += (weighted B)^T X.  The inputs b, c, x
// are bf16.  What has to keep 32 bits -- the state, and M and the weighted b, which carry decays and step sizes -- enters
// a product as the sum of two bf16 numbers, v = hi + lo, with a product for each (16 bits of mantissa, an error of 2^-17
// of the value); sums, decays and the state itself stay fp32.
//
// One block of eight warps per (head, request, slice of the values) walks the request's chunks.  Rows of the next chunk
// travel to shared memory (cp.async) while this one is computed, and one warp scans the next chunk's step sizes.  The
// state lives in the accumulators of the warps that own its tiles and is read back by all of them as a pair of bf16
// matrices in shared memory.  The walk starts from the state in the request's slot and leaves the new one there.
#include "common.cuh"

#ifndef TW_DK
#define TW_DK 128
#endif
#define SS_L 64                 // tokens of a chunk
#define SS_WARPS 8
#define SS_FLOOR (-58.0f)       // a token's log2 decay is held above this (2^-58): what it keeps of the state is below fp32 rounding

__device__ __forceinline__ void ss_ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ss_ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ss_ldm2t(uint32_t& r0, uint32_t& r1, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ss_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ss_copy16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;            // (0: the sixteen bytes are filled with zeros and nothing is read)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
// (x, y) as two pairs of bf16 whose sum is the pair to 16 bits
__device__ __forceinline__ void ss_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float ss_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct SsArgs {
    float* out;                                             // [rows, H * Dv]
    const __nv_bfloat16* q; const __nv_bfloat16* k; const __nv_bfloat16* v; int q_stride, k_stride, v_stride;
    const float* pre; int pre_stride;                       // projected step sizes [rows, H]
    const float* rate_log; const float* dt_bias; const float* skip;
    float* state; long long state_stride;
    const int* seq_slot; const int* seq_q_start; const int* seq_q_len;
    int H, Dv, qk_group, write_state;
};

// What the step sizes of a chunk give, in shared memory (log2 units for A).
struct SsScan {
    float cum[SS_L];        // A_t
    float dt[SS_L];         // dt_t, 0 behind the last token
    float in[SS_L];         // e^(A_t)
    float end[SS_L];        // e^(A_64 - A_s) dt_s
    float total;            // e^(A_64)
    float pad[3];
};

template <int DVS>          // values of the head that a block serves
__global__ void __launch_bounds__(32 * SS_WARPS, 1)
state_space_chunk_kernel(SsArgs a) {
    constexpr int N = TW_DK, MT = N / 16, NT = DVS / 8;
    constexpr int RS = N + 8, XS = DVS + 8;                 // padded row lengths: the eight rows of an ldmatrix fall into different banks
    constexpr int PARTS = MT >= SS_WARPS ? 1 : SS_WARPS / MT;       // warps that share a row tile of the state
    constexpr int MPW = MT >= SS_WARPS ? MT / SS_WARPS : 1;         // row tiles of the state per warp
    constexpr int NPW = NT >= PARTS ? NT / PARTS : 1;               // column tiles of the state per warp
    constexpr int YT = NT / 2 > 0 ? NT / 2 : 1;                     // column tiles of Y per warp
    constexpr int STAGE = 2 * SS_L * RS + SS_L * XS;                // bf16 values of a stage: C, B, X
    static_assert(N == 16 || N == 32 || N == 64 || N == 128 || N == 256, "state sizes");
    extern __shared__ __align__(16) unsigned char ss_smem[];
    __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(ss_smem);
    __nv_bfloat16* sh = stages + 2 * STAGE;                 // the state's hi [N][XS], then lo
    SsScan* scans = reinterpret_cast<SsScan*>(sh + 2 * N * XS);
    tw_grid_wait();
    tw_grid_launch_dependents();
    const int h = blockIdx.x, s = blockIdx.y, d0 = blockIdx.z * DVS;
    const int len = a.seq_q_len[s];
    if (len <= 0) return;
    const int start = a.seq_q_start[s];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, tq = lane & 3;
    const int chunks = (len + SS_L - 1) / SS_L;
    const __nv_bfloat16* gq = a.q + (size_t)start * a.q_stride + (h / a.qk_group) * N;
    const __nv_bfloat16* gk = a.k + (size_t)start * a.k_stride + (h / a.qk_group) * N;
    const __nv_bfloat16* gv = a.v + (size_t)start * a.v_stride + (size_t)h * a.Dv + d0;
    float* slot = a.state + (size_t)a.seq_slot[s] * a.state_stride + (size_t)h * N * a.Dv + d0;
    const uint32_t stage0 = (uint32_t)__cvta_generic_to_shared(stages), sh0 = (uint32_t)__cvta_generic_to_shared(sh);

    auto fetch = [&](int c) {           // the rows of chunk c into its stage
        const uint32_t base = stage0 + (uint32_t)((c & 1) * STAGE * 2);
        for (int e = tid; e < SS_L * (N / 8); e += 32 * SS_WARPS) {
            const int t = e / (N / 8), i = (e - t * (N / 8)) * 8, row = c * SS_L + t;
            const bool live = row < len;
            const size_t r = live ? row : 0;
            ss_copy16(base + (uint32_t)(t * RS + i) * 2, gq + r * a.q_stride + i, live);
            ss_copy16(base + (uint32_t)((SS_L + t) * RS + i) * 2, gk + r * a.k_stride + i, live);
        }
        for (int e = tid; e < SS_L * (DVS / 8); e += 32 * SS_WARPS) {
            const int t = e / (DVS / 8), i = (e - t * (DVS / 8)) * 8, row = c * SS_L + t;
            const bool live = row < len;
            ss_copy16(base + (uint32_t)(2 * SS_L * RS + t * XS + i) * 2, gv + (size_t)(live ? row : 0) * a.v_stride + i, live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // the scanning warp's step sizes, loaded a chunk before they are used
    const float rate = expf(a.rate_log[h]) * 1.4426950408889634f, bias = a.dt_bias[h], skip = a.skip[h];
    float raw0 = 0.f, raw1 = 0.f;
    auto load_steps = [&](int c) {
        const int r0 = c * SS_L + lane, r1 = r0 + 32;
        raw0 = r0 < len ? a.pre[(size_t)(start + r0) * a.pre_stride + h] : 0.f;
        raw1 = r1 < len ? a.pre[(size_t)(start + r1) * a.pre_stride + h] : 0.f;
    };
    auto scan_steps = [&](int c) {
        SsScan& sc = scans[c & 1];
        const int r0 = c * SS_L + lane, r1 = r0 + 32;
        const float t0 = r0 < len ? ss_softplus(raw0 + bias) : 0.f, t1 = r1 < len ? ss_softplus(raw1 + bias) : 0.f;
        float v0 = fmaxf(-rate * t0, SS_FLOOR), v1 = fmaxf(-rate * t1, SS_FLOOR);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u0 = __shfl_up_sync(0xffffffffu, v0, o), u1 = __shfl_up_sync(0xffffffffu, v1, o);
            if (lane >= o) { v0 += u0; v1 += u1; }
        }
        v1 += __shfl_sync(0xffffffffu, v0, 31);
        const float last = __shfl_sync(0xffffffffu, v1, 31);
        sc.cum[lane] = v0; sc.cum[lane + 32] = v1;
        sc.dt[lane] = t0; sc.dt[lane + 32] = t1;
        sc.in[lane] = exp2f(v0); sc.in[lane + 32] = exp2f(v1);
        sc.end[lane] = exp2f(last - v0) * t0; sc.end[lane + 32] = exp2f(last - v1) * t1;
        if (lane == 0) sc.total = exp2f(last);
    };

    // ---- the state's tiles of this warp: rows sm[i] .. + 15, columns 8 (sn + j)
    const int sm_first = MT >= SS_WARPS ? warp * MPW : warp % MT;
    const int sn = MT >= SS_WARPS ? 0 : (warp / MT) * NPW;
    const bool owns = sn < NT;
    float S[MPW][NPW][4];
    if (owns) {
#pragma unroll
        for (int i = 0; i < MPW; ++i)
#pragma unroll
            for (int j = 0; j < NPW; ++j) {
                const float* p = slot + (size_t)((sm_first + i) * 16 + g) * a.Dv + (sn + j) * 8 + 2 * tq;
                const float2 u = *reinterpret_cast<const float2*>(p), w = *reinterpret_cast<const float2*>(p + (size_t)8 * a.Dv);
                S[i][j][0] = u.x; S[i][j][1] = u.y; S[i][j][2] = w.x; S[i][j][3] = w.y;
            }
    }
    auto publish = [&]() {              // the state for everybody: hi and lo
        if (!owns) return;
#pragma unroll
        for (int i = 0; i < MPW; ++i)
#pragma unroll
            for (int j = 0; j < NPW; ++j) {
                const int at = ((sm_first + i) * 16 + g) * XS + (sn + j) * 8 + 2 * tq;
                uint32_t hi, lo;
                ss_split(S[i][j][0], S[i][j][1], hi, lo);
                *reinterpret_cast<uint32_t*>(sh + at) = hi;
                *reinterpret_cast<uint32_t*>(sh + N * XS + at) = lo;
                ss_split(S[i][j][2], S[i][j][3], hi, lo);
                *reinterpret_cast<uint32_t*>(sh + at + 8 * XS) = hi;
                *reinterpret_cast<uint32_t*>(sh + N * XS + at + 8 * XS) = lo;
            }
    };

    fetch(0);
    if (warp == 0) { load_steps(0); scan_steps(0); load_steps(1); }
    publish();
    // the rows of Y of this warp: the halves of the columns take the row tiles in opposite order, so that the four
    // schedulers of an SM get equal shares of the triangle
    const int half = warp >> 2, rt = half ? 3 - (warp & 3) : (warp & 3);
    const int yn = half * YT;
    const bool writes_y = yn < NT;

    for (int c = 0; c < chunks; ++c) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                // this chunk's rows, its scan and the state are there; the other stage is free
        if (c + 1 < chunks) {
            fetch(c + 1);
            if (warp == 0) { scan_steps(c + 1); load_steps(c + 2); }
        }
        const uint32_t cs = stage0 + (uint32_t)((c & 1) * STAGE * 2), bs = cs + SS_L * RS * 2, xs = bs + SS_L * RS * 2;
        const SsScan& sc = scans[c & 1];
        if (writes_y) {
            float G[SS_L / 8][4], Y[YT][4];
#pragma unroll
            for (int j = 0; j < SS_L / 8; ++j) G[j][0] = G[j][1] = G[j][2] = G[j][3] = 0.f;
#pragma unroll
            for (int j = 0; j < YT; ++j) Y[j][0] = Y[j][1] = Y[j][2] = Y[j][3] = 0.f;
#pragma unroll 2
            for (int k = 0; k < MT; ++k) {
                uint32_t A[4], B[4];
                ss_ldm4(A, cs + (uint32_t)((rt * 16 + (lane & 15)) * RS + k * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int j = 0; j < SS_L / 16; ++j) {
                    if (j <= rt) {      // tokens behind the row tile's last are not seen
                        ss_ldm4(B, bs + (uint32_t)((j * 16 + (lane & 7) + ((lane >> 4) << 3)) * RS + k * 16 + ((lane >> 3) & 1) * 8) * 2);
                        ss_mma(G[2 * j], A, B[0], B[1]);
                        ss_mma(G[2 * j + 1], A, B[2], B[3]);
                    }
                }
#pragma unroll
                for (int p = 0; p < 2; ++p) {           // hi, lo
                    const uint32_t base = sh0 + (uint32_t)(p * N * XS + (k * 16 + (lane & 15)) * XS) * 2;
                    if constexpr (YT % 2 == 0) {
#pragma unroll
                        for (int j = 0; j < YT; j += 2) {
                            ss_ldm4t(B, base + (uint32_t)((yn + j) * 8 + (lane >> 4) * 8) * 2);
                            ss_mma(Y[j], A, B[0], B[1]);
                            ss_mma(Y[j + 1], A, B[2], B[3]);
                        }
                    } else {
                        ss_ldm2t(B[0], B[1], base + (uint32_t)(yn * 8) * 2);
                        ss_mma(Y[0], A, B[0], B[1]);
                    }
                }
            }
            const int ta = rt * 16 + g, tb = ta + 8;
            const float ia = sc.in[ta], ib = sc.in[tb], ca = sc.cum[ta], cb = sc.cum[tb];
#pragma unroll
            for (int j = 0; j < YT; ++j) { Y[j][0] *= ia; Y[j][1] *= ia; Y[j][2] *= ib; Y[j][3] *= ib; }
#pragma unroll
            for (int j = 0; j < SS_L / 16; ++j) {
                if (j <= rt) {
                    uint32_t hi[4], lo[4];
#pragma unroll
                    for (int e = 0; e < 2; ++e) {       // the two column tiles of G are the two halves of the k of M
                        const int s0 = j * 16 + e * 8 + 2 * tq, s1 = s0 + 1;
                        const float2 cum = *reinterpret_cast<const float2*>(sc.cum + s0), dt = *reinterpret_cast<const float2*>(sc.dt + s0);
                        float m[4];
                        m[0] = s0 <= ta ? G[2 * j + e][0] * exp2f(ca - cum.x) * dt.x : 0.f;
                        m[1] = s1 <= ta ? G[2 * j + e][1] * exp2f(ca - cum.y) * dt.y : 0.f;
                        m[2] = s0 <= tb ? G[2 * j + e][2] * exp2f(cb - cum.x) * dt.x : 0.f;
                        m[3] = s1 <= tb ? G[2 * j + e][3] * exp2f(cb - cum.y) * dt.y : 0.f;
                        if (s0 == ta) m[0] += skip;
                        if (s1 == ta) m[1] += skip;
                        if (s0 == tb) m[2] += skip;
                        if (s1 == tb) m[3] += skip;
                        ss_split(m[0], m[1], hi[2 * e], lo[2 * e]);
                        ss_split(m[2], m[3], hi[2 * e + 1], lo[2 * e + 1]);
                    }
                    const uint32_t base = xs + (uint32_t)((j * 16 + (lane & 15)) * XS) * 2;
                    uint32_t B[4];
                    if constexpr (YT % 2 == 0) {
#pragma unroll
                        for (int n = 0; n < YT; n += 2) {
                            ss_ldm4t(B, base + (uint32_t)((yn + n) * 8 + (lane >> 4) * 8) * 2);
                            ss_mma(Y[n], hi, B[0], B[1]);
                            ss_mma(Y[n], lo, B[0], B[1]);
                            ss_mma(Y[n + 1], hi, B[2], B[3]);
                            ss_mma(Y[n + 1], lo, B[2], B[3]);
                        }
                    } else {
                        ss_ldm2t(B[0], B[1], base + (uint32_t)(yn * 8) * 2);
                        ss_mma(Y[0], hi, B[0], B[1]);
                        ss_mma(Y[0], lo, B[0], B[1]);
                    }
                }
            }
            const int ra = c * SS_L + ta, rb = ra + 8;
            float* oa = a.out + (size_t)(start + ra) * ((size_t)a.H * a.Dv) + (size_t)h * a.Dv + d0 + yn * 8 + 2 * tq;
            float* ob = oa + (size_t)8 * a.H * a.Dv;
#pragma unroll
            for (int j = 0; j < YT; ++j) {
                if (ra < len) *reinterpret_cast<float2*>(oa + j * 8) = make_float2(Y[j][0], Y[j][1]);
                if (rb < len) *reinterpret_cast<float2*>(ob + j * 8) = make_float2(Y[j][2], Y[j][3]);
            }
        }
        if (owns) {
            const float keep = sc.total;
#pragma unroll
            for (int i = 0; i < MPW; ++i)
#pragma unroll
                for (int j = 0; j < NPW; ++j) { S[i][j][0] *= keep; S[i][j][1] *= keep; S[i][j][2] *= keep; S[i][j][3] *= keep; }
#pragma unroll
            for (int k = 0; k < SS_L / 16; ++k) {
                const float2 wa = *reinterpret_cast<const float2*>(sc.end + k * 16 + 2 * tq);
                const float2 wb = *reinterpret_cast<const float2*>(sc.end + k * 16 + 8 + 2 * tq);
                uint32_t B[NPW][2];
                const uint32_t xbase = xs + (uint32_t)((k * 16 + (lane & 15)) * XS) * 2;
                if constexpr (NPW % 2 == 0) {
#pragma unroll
                    for (int j = 0; j < NPW; j += 2) {
                        uint32_t R[4];
                        ss_ldm4t(R, xbase + (uint32_t)((sn + j) * 8 + (lane >> 4) * 8) * 2);
                        B[j][0] = R[0]; B[j][1] = R[1]; B[j + 1][0] = R[2]; B[j + 1][1] = R[3];
                    }
                } else {
                    ss_ldm2t(B[0][0], B[0][1], xbase + (uint32_t)(sn * 8) * 2);
                }
#pragma unroll
                for (int i = 0; i < MPW; ++i) {
                    uint32_t R[4], hi[4], lo[4];
                    ss_ldm4t(R, bs + (uint32_t)((k * 16 + (lane & 7) + ((lane >> 4) << 3)) * RS + (sm_first + i) * 16 + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
                    for (int e = 0; e < 4; ++e) {       // registers 0, 1: the first eight tokens of the sixteen; 2, 3: the others
                        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&R[e]));
                        const float2 w = e < 2 ? wa : wb;
                        ss_split(f.x * w.x, f.y * w.y, hi[e], lo[e]);
                    }
#pragma unroll
                    for (int j = 0; j < NPW; ++j) {
                        ss_mma(S[i][j], hi, B[j][0], B[j][1]);
                        ss_mma(S[i][j], lo, B[j][0], B[j][1]);
                    }
                }
            }
        }
        __syncthreads();                // nobody reads the old state any more
        if (c + 1 < chunks) publish();
    }
    if (a.write_state && owns) {
#pragma unroll
        for (int i = 0; i < MPW; ++i)
#pragma unroll
            for (int j = 0; j < NPW; ++j) {
                float* p = slot + (size_t)((sm_first + i) * 16 + g) * a.Dv + (sn + j) * 8 + 2 * tq;
                *reinterpret_cast<float2*>(p) = make_float2(S[i][j][0], S[i][j][1]);
                *reinterpret_cast<float2*>(p + (size_t)8 * a.Dv) = make_float2(S[i][j][2], S[i][j][3]);
            }
    }
}

template <int DVS>
static int ss_launch(const SsArgs& a, int n_seqs, cudaStream_t stream) {
    constexpr int N = TW_DK, RS = N + 8, XS = DVS + 8;
    constexpr size_t smem = (2 * (size_t)(2 * SS_L * RS + SS_L * XS) + 2 * (size_t)N * XS) * 2 + 2 * sizeof(SsScan);
    static_assert(smem <= 227 * 1024, "shared memory");
    const cudaError_t e = cudaFuncSetAttribute(state_space_chunk_kernel<DVS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    return tw_launch(state_space_chunk_kernel<DVS>, dim3(a.H, n_seqs, a.Dv / DVS), dim3(32 * SS_WARPS), smem, stream, 1, a);
}

// q, k [rows, heads / qk_group * N], v [rows, heads * Dv] bf16 (column slices of wider rows on 16-byte boundaries); state
// [slots, state_stride] with a head's [N, Dv] at h * N * Dv.  `slice`: values of a head per block (64, 32 or 16).
TW_EXPORT int tw_state_space_chunks(float* out, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                                    const float* pre, int pre_stride, const float* rate_log, const float* dt_bias, const float* skip,
                                    float* state, long long state_stride, const int* seq_slot, const int* seq_q_start,
                                    const int* seq_q_len, int n_seqs, int H, int N, int Dv, int qk_group, int slice, int write_state,
                                    cudaStream_t stream) {
    if (n_seqs <= 0 || H <= 0) return 0;
    auto a16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (N != TW_DK || (slice != 64 && slice != 32 && slice != 16) || Dv <= 0 || Dv % slice || qk_group <= 0 || H % qk_group || (q_stride & 7)
        || (k_stride & 7) || (v_stride & 7) || !a16(q) || !a16(k) || !a16(v) || (state_stride & 1) || (reinterpret_cast<uintptr_t>(state) & 7)
        || (reinterpret_cast<uintptr_t>(out) & 7))
        return (int)cudaErrorInvalidValue;
    SsArgs a;
    a.out = out;
    a.q = (const __nv_bfloat16*)q; a.k = (const __nv_bfloat16*)k; a.v = (const __nv_bfloat16*)v;
    a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride;
    a.pre = pre; a.pre_stride = pre_stride; a.rate_log = rate_log; a.dt_bias = dt_bias; a.skip = skip;
    a.state = state; a.state_stride = state_stride;
    a.seq_slot = seq_slot; a.seq_q_start = seq_q_start; a.seq_q_len = seq_q_len;
    a.H = H; a.Dv = Dv; a.qk_group = qk_group; a.write_state = write_state;
    if (slice == 64) return ss_launch<64>(a, n_seqs, stream);
    if (slice == 32) return ss_launch<32>(a, n_seqs, stream);
    return ss_launch<16>(a, n_seqs, stream);
}
