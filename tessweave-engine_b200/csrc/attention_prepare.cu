// What a step's projected rows need before attention can read them, in one pass over each row:
//
//   row = [q: Hq heads of D | k: Hkv heads of D | v: Hkv heads of Dv | g: Hq numbers (optional)]
//
//   1. rotation by position of the first `rot_dims` values of every head of q and k (pairs of neighbours, or of halves
//      of the rotated part); angle = float(position) * inv_freq[i], cos and sin multiplied by `magnitude`;
//   2. the values of an earlier layer blended in (role 2): v <- (1 - lambda) v + lambda first, `first` the rows of
//      values that the layer with role 1 left for the later layers of the step;
//   3. q into rows of its own, k and v into the token's place in its request's pages, sigmoid(g) into fp32
//      [rows][Hq] for the attention kernels, which multiply each head's output by it.
//
// The source is the product's rows, or the fp32 slices of a product split over k, which are added here in the order
// that every consumer of a split product uses.  All arithmetic between the loads and the stores is fp32, each result
// is rounded once.  A block serves one token (or a share of its columns, in steps with few tokens); the cosines and
// sines of the position are made once per block and shared by all heads.
#include "common.cuh"

namespace {

struct PrepareArgs {
    int width;                   // columns of a row (and of a slice)
    int Hq, Hkv, D, Dv;
    int rot_dims, interleaved;
    float magnitude;
    const float* inv_freq;       // [rot_dims / 2]
    int v_role;                  // 0: values as projected; 1: and left for later layers in `first`; 2: blended with `first`
    const float* lambda;         // one number (role 2)
    float* gate;                 // fp32 [rows][Hq], or null: the row has no gate columns
    const int *positions, *seq_of_token, *seq_slot, *block_table;
    int table_stride, page_size, num_pages, write_cache;
    int* status;
};

// sums of `nsplit` slices of N neighbouring columns: whole groups of four slices into four sums by slice mod 4, the
// rest into the first, then (s0 + s1) + (s2 + s3)
template <int N>
__device__ __forceinline__ void sum_slices(const float* p, int nsplit, size_t stride, float (&out)[N]) {
    float s[4][N];
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int j = 0; j < N; ++j) s[u][j] = 0.f;
    int k = 0;
    for (; k + 4 <= nsplit; k += 4) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if constexpr (N == 8) {
                const float4 a = *reinterpret_cast<const float4*>(p + (size_t)(k + u) * stride);
                const float4 b = *reinterpret_cast<const float4*>(p + (size_t)(k + u) * stride + 4);
                s[u][0] += a.x; s[u][1] += a.y; s[u][2] += a.z; s[u][3] += a.w;
                s[u][4] += b.x; s[u][5] += b.y; s[u][6] += b.z; s[u][7] += b.w;
            } else {
                s[u][0] += p[(size_t)(k + u) * stride];
            }
        }
    }
    for (; k < nsplit; ++k) {
        if constexpr (N == 8) {
            const float4 a = *reinterpret_cast<const float4*>(p + (size_t)k * stride);
            const float4 b = *reinterpret_cast<const float4*>(p + (size_t)k * stride + 4);
            s[0][0] += a.x; s[0][1] += a.y; s[0][2] += a.z; s[0][3] += a.w;
            s[0][4] += b.x; s[0][5] += b.y; s[0][6] += b.z; s[0][7] += b.w;
        } else {
            s[0][0] += p[(size_t)k * stride];
        }
    }
#pragma unroll
    for (int j = 0; j < N; ++j) out[j] = (s[0][j] + s[1][j]) + (s[2][j] + s[3][j]);
}

__device__ __forceinline__ void load8(const float* p, float (&x)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&x)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h[e]);
        x[2 * e] = f.x; x[2 * e + 1] = f.y;
    }
}
__device__ __forceinline__ void store8(float* p, const float (&x)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(x[0], x[1], x[2], x[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(x[4], x[5], x[6], x[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&x)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// VEC: eight neighbouring columns per item (pairs of neighbours, head sizes that are multiples of 8, 16-byte aligned
// rows); otherwise a pair, or a single value that is not rotated, per item.  SLICES: `partial` is the source.
template <typename T, bool VEC, bool SLICES>
__global__ void __launch_bounds__(256)
attention_prepare_kernel(T* __restrict__ q_out, const T* __restrict__ rows, int row_stride, const float* __restrict__ partial,
                         int nsplit, size_t split_stride, T* first, T* __restrict__ k_cache, T* __restrict__ v_cache,
                         const PrepareArgs a) {
    extern __shared__ float2 turn[];                 // [rot_dims / 2] (cos, sin) of this token's position
    // which request and place a row belongs to is known before the step's first kernel starts
    const int n = blockIdx.x;
    const int s = a.seq_of_token[n];
    const int pos = a.positions[n];
    const int blk = pos / a.page_size, in_page = pos - blk * a.page_size;
    const int page = (s >= 0 && a.write_cache && blk < a.table_stride) ? a.block_table[(size_t)a.seq_slot[s] * a.table_stride + blk] : -1;
    const int half = a.rot_dims >> 1;
    if (s >= 0) {
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            float sn, cs;
            sincosf((float)pos * a.inv_freq[i], &sn, &cs);
            turn[i] = make_float2(cs * a.magnitude, sn * a.magnitude);
        }
    }
    __syncthreads();
    tw_grid_wait();
    tw_grid_launch_dependents();
    if (s < 0) return;
    const bool store = a.write_cache && page >= 0 && page < a.num_pages;
    if (a.write_cache && !store && threadIdx.x == 0) atomicOr(a.status, TW_ERR_PAGE);
    const T* row = rows + (size_t)n * row_stride;
    const float* prow = partial ? partial + (size_t)n * a.width : nullptr;
    const float lam = a.v_role == 2 ? *a.lambda : 0.f;
    const int D = a.D, Dv = a.Dv, q_size = a.Hq * D, k_size = a.Hkv * D, v_size = a.Hkv * Dv;
    const int at = blockIdx.y * blockDim.x + threadIdx.x, step = gridDim.y * blockDim.x;
    if constexpr (VEC) {
        const int n8 = (q_size + k_size + v_size) >> 3;
        // rows: the loads of up to three items go out before the first store (one round trip to memory, not three)
        constexpr int AHEAD = SLICES ? 1 : 3, RAW = sizeof(T) / 2;
        for (int base = at; base < n8; base += AHEAD * step) {
            uint4 raw[AHEAD][RAW];
            if constexpr (!SLICES) {
#pragma unroll
                for (int j = 0; j < AHEAD; ++j) {
                    const int item = base + j * step;
#pragma unroll
                    for (int r = 0; r < RAW; ++r)
                        raw[j][r] = item < n8 ? __ldg(reinterpret_cast<const uint4*>(row + (item << 3)) + r) : make_uint4(0u, 0u, 0u, 0u);
                }
            }
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int item = base + j * step;
                if (item >= n8) break;
                const int col = item << 3;
                float x[8];
                if constexpr (SLICES) sum_slices<8>(prow + col, nsplit, split_stride, x);
                else load8(reinterpret_cast<const T*>(&raw[j][0]), x);
                if (col < q_size + k_size) {
                    const int c = col < q_size ? col : col - q_size;
                    const int head = c / D, d = c - head * D;
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        if (d + 2 * e < a.rot_dims) {
                            const float2 t = turn[(d >> 1) + e];
                            const float u = x[2 * e], v = x[2 * e + 1];
                            x[2 * e] = u * t.x - v * t.y;
                            x[2 * e + 1] = v * t.x + u * t.y;
                        }
                    }
                    if (col < q_size) store8(q_out + (size_t)n * q_size + col, x);
                    else if (store) store8(k_cache + (((size_t)page * a.Hkv + head) * a.page_size + in_page) * D + d, x);
                } else {
                    const int c = col - q_size - k_size;
                    const int head = c / Dv, d = c - head * Dv;
                    if (a.v_role == 2) {
                        float f[8];
                        load8(first + (size_t)n * v_size + c, f);
#pragma unroll
                        for (int e = 0; e < 8; ++e) x[e] = (1.f - lam) * x[e] + lam * f[e];
                    } else if (a.v_role == 1) {
                        store8(first + (size_t)n * v_size + c, x);
                    }
                    if (store) store8(v_cache + (((size_t)page * a.Hkv + head) * a.page_size + in_page) * Dv + d, x);
                }
            }
        }
    } else {
        auto load1 = [&](int col) -> float {
            if constexpr (!SLICES) return tw_to_float(row[col]);
            float x[1];
            sum_slices<1>(prow + col, nsplit, split_stride, x);
            return x[0];
        };
        const int per_head = D - half;               // half pairs and D - rot_dims singles
        const int qk_items = (a.Hq + a.Hkv) * per_head;
        for (int item = at; item < qk_items + v_size; item += step) {
            if (item < qk_items) {
                const int head = item / per_head, i = item - head * per_head;
                const bool is_q = head < a.Hq;
                T* dst = is_q ? q_out + (size_t)n * q_size + head * D
                              : (store ? k_cache + (((size_t)page * a.Hkv + (head - a.Hq)) * a.page_size + in_page) * D : nullptr);
                if (i < half) {
                    const int d0 = a.interleaved ? 2 * i : i, d1 = a.interleaved ? 2 * i + 1 : i + half;
                    const float u = load1(head * D + d0), v = load1(head * D + d1);
                    const float2 t = turn[i];
                    if (dst) {
                        dst[d0] = tw_from_float<T>(u * t.x - v * t.y);
                        dst[d1] = tw_from_float<T>(v * t.x + u * t.y);
                    }
                } else if (dst) {
                    dst[i + half] = tw_from_float<T>(load1(head * D + i + half));
                }
            } else {
                const int c = item - qk_items;
                const int head = c / Dv, d = c - head * Dv;
                float x = load1(q_size + k_size + c);
                if (a.v_role == 2) x = (1.f - lam) * x + lam * tw_to_float(first[(size_t)n * v_size + c]);
                else if (a.v_role == 1) first[(size_t)n * v_size + c] = tw_from_float<T>(x);
                if (store) v_cache[(((size_t)page * a.Hkv + head) * a.page_size + in_page) * Dv + d] = tw_from_float<T>(x);
            }
        }
    }
    if (a.gate) {
        const int g_col = q_size + k_size + v_size;
        for (int h = at; h < a.Hq; h += step) {
            float z[1];
            if constexpr (SLICES) sum_slices<1>(prow + g_col + h, nsplit, split_stride, z);
            else z[0] = tw_to_float(row[g_col + h]);
            a.gate[(size_t)n * a.Hq + h] = 1.f / (1.f + expf(-z[0]));
        }
    }
}

template <typename T, bool VEC>
int launch(void* q_out, const void* rows, int row_stride, const float* partial, int nsplit, long split_stride, void* first,
           void* k_cache, void* v_cache, const PrepareArgs& a, int n_tokens, int items, cudaStream_t stream) {
    // few tokens: a row's columns are shared by several blocks, so that the step does not wait for a handful of SMs
    int parts = (items + 255) / 256;
    const int room = (2 * 148 + n_tokens - 1) / n_tokens;
    if (parts > room) parts = room;
    if (parts < 1) parts = 1;
    auto kernel = partial ? attention_prepare_kernel<T, VEC, true> : attention_prepare_kernel<T, VEC, false>;
    return tw_launch(kernel, dim3(n_tokens, parts), dim3(256), (size_t)(a.rot_dims / 2) * sizeof(float2),
                     stream, 1, (T*)q_out, (const T*)rows, row_stride, partial, nsplit, (size_t)split_stride, (T*)first,
                     (T*)k_cache, (T*)v_cache, a);
}

}  // namespace

// `rows` [n_tokens, row_stride] or, when `partial` is given, fp32 slices [nsplit][rows][width], `split_stride` floats
// apart.  q_out: contiguous [n_tokens, Hq * D].  `first`: contiguous [n_tokens, Hkv * Dv] (v_role 1 writes it, 2 reads it).
TW_EXPORT int tw_attention_prepare(void* q_out, const void* rows, int row_stride, const float* partial, int nsplit, long split_stride,
                                   int width, int n_tokens, int Hq, int Hkv, int D, int Dv, int rot_dims, int interleaved,
                                   float magnitude, const float* inv_freq, int v_role, const float* lambda, void* first, float* gate,
                                   const int* positions, const int* seq_of_token, const int* seq_slot, const int* block_table,
                                   int table_stride, void* k_cache, void* v_cache, int page_size, int num_pages, int write_cache,
                                   int dtype, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (Hq <= 0 || Hkv <= 0 || D <= 0 || Dv <= 0 || rot_dims < 0 || (rot_dims & 1) || rot_dims > D || rot_dims > 4096 ||
        (rot_dims && !inv_freq) || v_role < 0 || v_role > 2 || (v_role && !first) || (v_role == 2 && !lambda) || page_size <= 0 ||
        (partial ? nsplit < 1 : !rows) || (long)width < (long)Hq * D + (long)Hkv * (D + Dv) + (gate ? Hq : 0))
        return (int)cudaErrorInvalidValue;
    const PrepareArgs a{width, Hq, Hkv, D, Dv, rot_dims, interleaved, magnitude, inv_freq, v_role, lambda, gate, positions,
                        seq_of_token, seq_slot, block_table, table_stride, page_size, num_pages, write_cache, status};
    auto a16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = (interleaved || rot_dims == 0) && (D & 7) == 0 && (Dv & 7) == 0 && a16(q_out) && a16(first) && a16(k_cache) &&
                     a16(v_cache) && (partial ? (a16(partial) && (width & 3) == 0 && (split_stride & 3) == 0)
                                              : (a16(rows) && (row_stride & (dtype == TW_F32 ? 3 : 7)) == 0));
    const int items = vec ? (Hq * D + Hkv * (D + Dv)) / 8 : (Hq + Hkv) * (D - rot_dims / 2) + Hkv * Dv;
    if (dtype == TW_F32)
        return vec ? launch<float, true>(q_out, rows, row_stride, partial, nsplit, split_stride, first, k_cache, v_cache, a, n_tokens, items, stream)
                   : launch<float, false>(q_out, rows, row_stride, partial, nsplit, split_stride, first, k_cache, v_cache, a, n_tokens, items, stream);
    return vec ? launch<__nv_bfloat16, true>(q_out, rows, row_stride, partial, nsplit, split_stride, first, k_cache, v_cache, a, n_tokens, items, stream)
               : launch<__nv_bfloat16, false>(q_out, rows, row_stride, partial, nsplit, split_stride, first, k_cache, v_cache, a, n_tokens, items, stream);
}
