// Linear attention of prompts with one decay a head, as products of tiles in float32 (linear_attention.cu has the recurrence itself).
//
// A sequence's tokens are cut into chunks of up to 64.  With a the head's decay, n the chunk's tokens, t and s places in it:
//   contribution of a chunk to the state      L = sum_s a^(n-1-s) k_s v_s^T                                    [D, Dv]
//   its outputs, from the incoming state S    o_t = a^(t+1) S^T q_t + sum_{s <= t} a^(t-s) (q_t . k_s) v_s     [n, Dv]
// Walking the tokens costs two multiply-adds an element of the state and token in the first and three in the second; as products it is
// one and one, plus 64 a token and entry of q and v.  All sums are float32 multiply-adds; the powers of a are worked out in float64.
// Queries, keys (and values, in float32) go through their activation and scale while they are brought to shared memory.
#include "linear_attention.cuh"

#define LT_THREADS 256

template <typename T>
__device__ __forceinline__ float4 lt_load4(const T* p, int left, bool vec) {          // up to four entries, zeros behind `left`
    if (vec && left >= 4) {
        if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4*>(p);
        else {
            const uint2 r = *reinterpret_cast<const uint2*>(p);
            const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
            return make_float4(a.x, a.y, b.x, b.y);
        }
    }
    return make_float4(left > 0 ? to_f(p[0]) : 0.f, left > 1 ? to_f(p[1]) : 0.f, left > 2 ? to_f(p[2]) : 0.f, left > 3 ? to_f(p[3]) : 0.f);
}
template <bool FAST>
__device__ __forceinline__ float4 lt_act4(float4 v, int act, float scale) {
    if (act) { v.x = la_act<FAST>(v.x, act); v.y = la_act<FAST>(v.y, act); v.z = la_act<FAST>(v.z, act); v.w = la_act<FAST>(v.w, act); }
    return make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
}
// acc += a * b on four entries, two multiply-adds an instruction (fma.rn.f32x2: each half rounds as a plain one does)
__device__ __forceinline__ void lt_fma4(float4& acc, float a, const float4& b) {
    asm("{\n\t.reg .b64 pa, b0, b1, c0, c1;\n\t"
        "mov.b64 pa, {%4, %4};\n\tmov.b64 b0, {%5, %6};\n\tmov.b64 b1, {%7, %8};\n\tmov.b64 c0, {%0, %1};\n\tmov.b64 c1, {%2, %3};\n\t"
        "fma.rn.f32x2 c0, pa, b0, c0;\n\tfma.rn.f32x2 c1, pa, b1, c1;\n\t"
        "mov.b64 {%0, %1}, c0;\n\tmov.b64 {%2, %3}, c1;\n\t}"
        : "+f"(acc.x), "+f"(acc.y), "+f"(acc.z), "+f"(acc.w) : "f"(a), "f"(b.x), "f"(b.y), "f"(b.z), "f"(b.w));
}

// pw[i] = a^i for i <= 64 (a^0 = 1, also for a = 0)
__device__ __forceinline__ void lt_powers(float* pw, float a) {
    const int i = threadIdx.x;
    if (i <= LA_CHUNK) {
        double r = 1.0, b = (double)a;
        for (int e = i; e; e >>= 1) { if (e & 1) r *= b; b *= b; }
        pw[i] = (float)r;
    }
}

// A thread's share of [64][TW] entries of a chunk (columns c0 .. of every token's run at `src`), zeros behind its tokens and behind the
// head's columns: all of it is asked for before any of it is used.
template <typename T, int TW>
struct LTRows {
    static constexpr int N = LA_CHUNK * TW / 4 / LT_THREADS;
    float4 v[N];
    __device__ __forceinline__ void load(const T* src, int ld, int n, int left, bool vec) {
#pragma unroll
        for (int e = 0; e < N; ++e) {
            const int i = threadIdx.x + e * LT_THREADS, t = i / (TW / 4), c = (i % (TW / 4)) * 4;
            v[e] = t < n ? lt_load4(src + (size_t)t * ld + c, left - c, vec) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    template <bool FAST, typename Scale>
    __device__ __forceinline__ void store(float* dst, int act, Scale scale) const {
#pragma unroll
        for (int e = 0; e < N; ++e) {
            const int i = threadIdx.x + e * LT_THREADS, t = i / (TW / 4);
            *reinterpret_cast<float4*>(dst + 4 * i) = lt_act4<FAST>(v[e], act, scale(t));
        }
    }
};
// Sixteen by sixteen threads: a warp is four by eight of them, so that what it reads of either operand is a few neighbouring runs.
__device__ __forceinline__ void lt_place(int& ty, int& tx) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    ty = (warp >> 1) * 4 + (lane >> 3);
    tx = (warp & 1) * 8 + (lane & 7);
}

// A block: one chunk, one head, TD x TV entries of L; thread (ty, tx) the rows ty * 4 + 64 j + 0..3 and columns tx * 4 + 64 j + 0..3.
template <typename T, typename TQ, int RD, int RV>
__global__ void __launch_bounds__(LT_THREADS) lt_contribution_kernel(LAArgs a, int tiles_d, int vec_q, int vec_v) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int TD = 16 * RD, TV = 16 * RV;
    constexpr bool FAST = sizeof(T) == 2;
    extern __shared__ __align__(16) float lt_smem[];
    float* ks = lt_smem;                                  // [64][TD]
    float* vs = ks + LA_CHUNK * TD;                       // [64][TV]
    __shared__ float pw[LA_CHUNK + 1];
    const int tid = threadIdx.x, h = blockIdx.y;
    int ty, tx, row, first, n;
    lt_place(ty, tx);
    const int d0 = (blockIdx.z % tiles_d) * TD, c0 = (blockIdx.z / tiles_d) * TV;
    la_find_chunk(a.row_first, a.row_lens, a.B, blockIdx.x, row, first, n);
    if (n <= 0) return;
    LTRows<TQ, TD> k_rows;
    LTRows<T, TV> v_rows;
    k_rows.load((const TQ*)a.qk + (size_t)first * a.qk_ld + a.k_off + h * a.D + d0, a.qk_ld, n, a.D - d0, vec_q);
    v_rows.load((const T*)a.proj + (size_t)first * a.ld + a.v_off + h * a.Dv + c0, a.ld, n, a.Dv - c0, vec_v);
    lt_powers(pw, a.head_decay[h]);
    __syncthreads();
    k_rows.template store<FAST>(ks, a.act_qk, [&](int t) { return t < n ? pw[n - 1 - t] : 0.f; });
    v_rows.template store<FAST>(vs, a.act_v, [](int) { return 1.f; });
    __syncthreads();
    float4 acc[RD][RV / 4];
#pragma unroll
    for (int i = 0; i < RD; ++i)
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) acc[i][j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
        float4 v[RV / 4];
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) v[j] = *reinterpret_cast<const float4*>(vs + t * TV + tx * 4 + 64 * j);
#pragma unroll
        for (int i = 0; i < RD / 4; ++i) {
            const float4 k = *reinterpret_cast<const float4*>(ks + t * TD + ty * 4 + 64 * i);
#pragma unroll
            for (int j = 0; j < RV / 4; ++j) {
                lt_fma4(acc[4 * i + 0][j], k.x, v[j]); lt_fma4(acc[4 * i + 1][j], k.y, v[j]);
                lt_fma4(acc[4 * i + 2][j], k.z, v[j]); lt_fma4(acc[4 * i + 3][j], k.w, v[j]);
            }
        }
    }
    float* dst = a.chunk_state + ((size_t)blockIdx.x * a.H + h) * a.D * a.Dv;
    const bool vec = a.Dv % 4 == 0;
#pragma unroll
    for (int i = 0; i < RD; ++i) {
        const int d = d0 + ty * 4 + 64 * (i / 4) + i % 4;
        if (d >= a.D) continue;
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) {
            const int c = c0 + tx * 4 + 64 * j;
            float* p = dst + (size_t)d * a.Dv + c;
            const float4 v = acc[i][j];
            if (vec && c + 4 <= a.Dv) *reinterpret_cast<float4*>(p) = v;
            else { if (c < a.Dv) p[0] = v.x; if (c + 1 < a.Dv) p[1] = v.y; if (c + 2 < a.Dv) p[2] = v.z; if (c + 3 < a.Dv) p[3] = v.w; }
        }
    }
    if (blockIdx.z == 0)
        for (int d = tid; d < a.D; d += LT_THREADS) a.chunk_decay[((size_t)blockIdx.x * a.H + h) * a.D + d] = pw[n];
}

#define LT_ROWS 32          // rows of the incoming state in shared memory at a time, two buffers

// A block: one chunk, one head, TV columns of its outputs; thread (ty, tx) the tokens ty * 4 + 0..3 and columns tx * 4 + 64 j + 0..3.
template <typename T, typename TQ, int RV>
__global__ void __launch_bounds__(LT_THREADS, 2) lt_output_kernel(LAArgs a, int DP, int vec_q, int vec_v) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int TV = 16 * RV, C = LA_CHUNK;
    constexpr bool FAST = sizeof(T) == 2;
    extern __shared__ __align__(16) float lt_smem[];
    float* qt = lt_smem;                                  // [DP][64]: queries, entry by entry
    float* pt = qt + DP * C;                              // [64 s][64 t]: weights of the chunk's own keys
    float* vs = pt + C * C;                               // [64][TV]
    float* kt = vs + C * TV;                              // [DP][64]: keys; afterwards two buffers of LT_ROWS rows of the state
    __shared__ float pw[C + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, c0 = blockIdx.z * TV;
    int ty, tx, row, first, n;
    lt_place(ty, tx);
    la_find_chunk(a.row_first, a.row_lens, a.B, blockIdx.x, row, first, n);
    if (n <= 0) return;
    LTRows<T, TV> v_rows;
    v_rows.load((const T*)a.proj + (size_t)first * a.ld + a.v_off + h * a.Dv + c0, a.ld, n, a.Dv - c0, vec_v);
    lt_powers(pw, a.head_decay[h]);
    // a lane a token: four entries are read as a run and stored to four columns, neighbouring lanes side by side
#pragma unroll 4
    for (int u = warp; u < 2 * (DP / 4); u += LT_THREADS / 32) {
        const int t = (u & 1) * 32 + lane, d = (u >> 1) * 4;
        float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
        if (t < n) {
            const TQ* p = (const TQ*)a.qk + (size_t)(first + t) * a.qk_ld + h * a.D + d;
            q = lt_act4<FAST>(lt_load4(p + a.q_off, a.D - d, vec_q), a.act_qk, a.q_scale);
            k = lt_act4<FAST>(lt_load4(p + a.k_off, a.D - d, vec_q), a.act_qk, 1.f);
        }
        qt[(d + 0) * C + t] = q.x; qt[(d + 1) * C + t] = q.y; qt[(d + 2) * C + t] = q.z; qt[(d + 3) * C + t] = q.w;
        kt[(d + 0) * C + t] = k.x; kt[(d + 1) * C + t] = k.y; kt[(d + 2) * C + t] = k.z; kt[(d + 3) * C + t] = k.w;
    }
    v_rows.template store<FAST>(vs, a.act_v, [](int) { return 1.f; });
    __syncthreads();
    {
        float4 w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int d = 0; d < DP; ++d) {
            const float4 q = *reinterpret_cast<const float4*>(qt + d * C + ty * 4), k = *reinterpret_cast<const float4*>(kt + d * C + tx * 4);
            lt_fma4(w[0], k.x, q); lt_fma4(w[1], k.y, q); lt_fma4(w[2], k.z, q); lt_fma4(w[3], k.w, q);       // w[s]: four tokens t
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int s = tx * 4 + i, t = ty * 4;
            float4 p;
            p.x = s <= t ? w[i].x * pw[t - s] : 0.f;
            p.y = s <= t + 1 ? w[i].y * pw[t + 1 - s] : 0.f;
            p.z = s <= t + 2 ? w[i].z * pw[t + 2 - s] : 0.f;
            p.w = s <= t + 3 ? w[i].w * pw[t + 3 - s] : 0.f;
            *reinterpret_cast<float4*>(pt + s * C + t) = p;
        }
    }
    __syncthreads();                                      // the keys' place is free, the weights are there
    float4 acc[4][RV / 4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) acc[i][j] = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* state = a.chunk_state + ((size_t)blockIdx.x * a.H + h) * a.D * a.Dv + c0;
    const bool vec_s = a.Dv % 4 == 0;
    auto bring = [&](int d0, float* to) {                 // rows d0 .. d0 + LT_ROWS of the incoming state
        for (int i = tid; i < LT_ROWS * TV / 4; i += LT_THREADS) {
            const int r = i / (TV / 4), c = (i % (TV / 4)) * 4;
            float* dst = to + r * TV + c;
            const float* src = state + (size_t)(d0 + r) * a.Dv + c;
            if (d0 + r < a.D && vec_s && c0 + c + 4 <= a.Dv) {
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
            } else *reinterpret_cast<float4*>(dst) = d0 + r < a.D ? lt_load4(src, a.Dv - c0 - c, false) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    bring(0, kt);
    for (int d0 = 0, b = 0; d0 < DP; d0 += LT_ROWS, b ^= 1) {
        if (d0 + LT_ROWS < DP) {
            bring(d0 + LT_ROWS, kt + (b ^ 1) * LT_ROWS * TV);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float* rows = kt + b * LT_ROWS * TV;
        const int m = min(LT_ROWS, DP - d0);
#pragma unroll 4
        for (int r = 0; r < m; ++r) {
            const float4 q = *reinterpret_cast<const float4*>(qt + (d0 + r) * C + ty * 4);
#pragma unroll
            for (int j = 0; j < RV / 4; ++j) {
                const float4 s = *reinterpret_cast<const float4*>(rows + r * TV + tx * 4 + 64 * j);
                lt_fma4(acc[0][j], q.x, s); lt_fma4(acc[1][j], q.y, s); lt_fma4(acc[2][j], q.z, s); lt_fma4(acc[3][j], q.w, s);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float p = pw[ty * 4 + i + 1];
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) { acc[i][j].x *= p; acc[i][j].y *= p; acc[i][j].z *= p; acc[i][j].w *= p; }
    }
    const int last = min(n, 16 * (warp >> 1) + 16);       // a warp's tokens are sixteen neighbours: later keys have no weight
#pragma unroll 4
    for (int s = 0; s < last; ++s) {
        const float4 p = *reinterpret_cast<const float4*>(pt + s * C + ty * 4);
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) {
            const float4 v = *reinterpret_cast<const float4*>(vs + s * TV + tx * 4 + 64 * j);
            lt_fma4(acc[0][j], p.x, v); lt_fma4(acc[1][j], p.y, v); lt_fma4(acc[2][j], p.z, v); lt_fma4(acc[3][j], p.w, v);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < RV / 4; ++j) {
            const int c = c0 + tx * 4 + 64 * j;
            float* p = a.out + (size_t)(first + t) * ((size_t)a.H * a.Dv) + (size_t)h * a.Dv + c;
            const float4 v = acc[i][j];
            if (vec_s && c + 4 <= a.Dv) *reinterpret_cast<float4*>(p) = v;
            else { if (c < a.Dv) p[0] = v.x; if (c + 1 < a.Dv) p[1] = v.y; if (c + 2 < a.Dv) p[2] = v.z; if (c + 3 < a.Dv) p[3] = v.w; }
        }
    }
}

// Whether runs of four entries can be read at once.
static int lt_vec(const void* p, size_t element, int ld, int off0, int off1, int size) {
    return ((uintptr_t)p & (4 * element - 1)) == 0 && ld % 4 == 0 && off0 % 4 == 0 && off1 % 4 == 0 && size % 4 == 0;
}

template <typename T, typename TQ, int RD, int RV>
static int lt_contributions(const LAArgs& a, cudaStream_t s) {
    const int td = (a.D + 16 * RD - 1) / (16 * RD), tv = (a.Dv + 16 * RV - 1) / (16 * RV);
    const size_t smem = (size_t)LA_CHUNK * 16 * (RD + RV) * 4;
    auto kernel = lt_contribution_kernel<T, TQ, RD, RV>;
    PE_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PE_TRY(pe_launch(kernel, dim3(a.max_chunks, a.H, td * tv), LT_THREADS, smem, s, a, td, lt_vec(a.qk, sizeof(TQ), a.qk_ld, a.q_off, a.k_off, a.D),
                     lt_vec(a.proj, sizeof(T), a.ld, a.v_off, 0, a.Dv)));
    PE_LAUNCH_CHECK();
    return 0;
}

template <typename T, typename TQ, int RV>
static int lt_outputs(const LAArgs& a, cudaStream_t s) {
    const int DP = (a.D + 3) / 4 * 4, tv = (a.Dv + 16 * RV - 1) / (16 * RV);
    const int keys = DP * LA_CHUNK, rows = 2 * LT_ROWS * 16 * RV;
    const size_t smem = ((size_t)DP * LA_CHUNK + LA_CHUNK * LA_CHUNK + LA_CHUNK * 16 * RV + (keys > rows ? keys : rows)) * 4;
    auto kernel = lt_output_kernel<T, TQ, RV>;
    PE_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PE_TRY(pe_launch(kernel, dim3(a.max_chunks, a.H, tv), LT_THREADS, smem, s, a, DP, lt_vec(a.qk, sizeof(TQ), a.qk_ld, a.q_off, a.k_off, a.D),
                     lt_vec(a.proj, sizeof(T), a.ld, a.v_off, 0, a.Dv)));
    PE_LAUNCH_CHECK();
    return 0;
}

template <typename T, typename TQ>
static int lt_contributions_by_size(const LAArgs& a, cudaStream_t s) {
    if (a.D > 64) return a.Dv > 64 ? lt_contributions<T, TQ, 8, 8>(a, s) : lt_contributions<T, TQ, 8, 4>(a, s);
    return a.Dv > 64 ? lt_contributions<T, TQ, 4, 8>(a, s) : lt_contributions<T, TQ, 4, 4>(a, s);
}

int la_tiles_contributions(const LAArgs& a, int types, cudaStream_t s) {
    if (a.D > 256) return PE_ERR_UNSUPPORTED;
    if (types == 0) return lt_contributions_by_size<float, float>(a, s);
    return types == 1 ? lt_contributions_by_size<bf16, bf16>(a, s) : lt_contributions_by_size<bf16, float>(a, s);
}

int la_tiles_outputs(const LAArgs& a, int types, cudaStream_t s) {
    if (a.D > 256) return PE_ERR_UNSUPPORTED;
    const bool wide = a.Dv > 64;
    if (types == 0) return wide ? lt_outputs<float, float, 8>(a, s) : lt_outputs<float, float, 4>(a, s);
    if (types == 1) return wide ? lt_outputs<bf16, bf16, 8>(a, s) : lt_outputs<bf16, bf16, 4>(a, s);
    return wide ? lt_outputs<bf16, float, 8>(a, s) : lt_outputs<bf16, float, 4>(a, s);
}
