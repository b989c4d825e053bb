// What lies between two blocks whose sublayers are added to the residual stream together: up to three terms, each optionally times a
// number per token and a vector over the columns, added to the 32-bit stream, and the RMS norm that the next block begins with.
#include "common.cuh"

namespace lb {

// One term of the sum.  Its value at (row, d) is given as one of
//   rows      [tokens, dim] of the activation type
//   partials  a product left as the partial sums of its K slices, [slices][tokens, dim] in 32-bit, `slice_stride` floats apart, added in
//             slice order and rounded to the activation type as the product's own epilogue would have stored it
//   pair_out  the routed experts' outputs, [tokens * top, dim] in 32-bit: the sum over a token's pairs whose expert exists, in the order of
//             the choice, each times pair_weight (null: 1)
// and it counts gate[row * gate_stride] (null: 1) * scale[d] (null: 1) times.
struct ResidualTerm {
    const void* rows;
    const float* partials;
    const float* pair_out;
    const float* pair_weight;
    const int* pair_expert;
    const float* gate;
    const float* scale;
    long long slice_stride;
    int slices, top, experts, gate_stride;
};

constexpr int kMaxTerms = 3;
struct ResidualTerms {
    ResidualTerm term[kMaxTerms];
    int count;
};

template <typename T>
__device__ __forceinline__ float4 load_four(const T* address) {
    if constexpr (sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(address);
        const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(low.x, low.y, high.x, high.y);
    } else {
        return *reinterpret_cast<const float4*>(address);
    }
}

template <typename T>
__device__ __forceinline__ void store_four(T* address, float4 v) {
    if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162 low = __floats2bfloat162_rn(v.x, v.y), high = __floats2bfloat162_rn(v.z, v.w);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&low);
        packed.y = *reinterpret_cast<const uint32_t*>(&high);
        *reinterpret_cast<uint2*>(address) = packed;
    } else {
        *reinterpret_cast<float4*>(address) = v;
    }
}

__device__ __forceinline__ void add_scaled(float4& to, float factor, float4 v) {
    to.x += factor * v.x;
    to.y += factor * v.y;
    to.z += factor * v.z;
    to.w += factor * v.w;
}

// Four neighbouring columns of a term (before its gate and scale).
template <typename T>
__device__ __forceinline__ float4 term_value(const ResidualTerm& term, size_t row, int d, int dim) {
    if (term.rows != nullptr) return load_four(static_cast<const T*>(term.rows) + row * dim + d);
    float4 total = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (term.partials != nullptr) {
        const float* mine = term.partials + row * dim + d;
        for (int s = 0; s < term.slices; s += 4) {   // four slices' loads leave before the first is added (the order of the additions stays)
            float4 part[4];
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (s + u < term.slices) part[u] = __ldcs(reinterpret_cast<const float4*>(mine + static_cast<size_t>(s + u) * term.slice_stride));
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (s + u < term.slices) add_scaled(total, 1.0f, part[u]);
        }
        return make_float4(round_to<T>(total.x), round_to<T>(total.y), round_to<T>(total.z), round_to<T>(total.w));
    }
    for (int k0 = 0; k0 < term.top; k0 += 4) {   // likewise four experts' loads
        float4 part[4];
        float weight[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const size_t pair = row * term.top + k0 + u;
            const int expert = k0 + u < term.top ? term.pair_expert[pair] : -1;
            const bool real = expert >= 0 && expert < term.experts;   // rows of pairs without an expert were never written
            weight[u] = real && term.pair_weight != nullptr ? term.pair_weight[pair] : 1.0f;
            part[u] = real ? *reinterpret_cast<const float4*>(term.pair_out + pair * dim + d) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) add_scaled(total, weight[u], part[u]);
    }
    return total;
}

// One column, for widths that are no multiple of four.
template <typename T>
__device__ __forceinline__ float term_value_one(const ResidualTerm& term, size_t row, int d, int dim) {
    if (term.rows != nullptr) return to_float(static_cast<const T*>(term.rows)[row * dim + d]);
    float total = 0.0f;
    if (term.partials != nullptr) {
        for (int s = 0; s < term.slices; ++s) total += term.partials[static_cast<size_t>(s) * term.slice_stride + row * dim + d];
        return round_to<T>(total);
    }
    for (int k = 0; k < term.top; ++k) {
        const size_t pair = row * term.top + k;
        const int expert = term.pair_expert[pair];
        if (expert >= 0 && expert < term.experts) total += (term.pair_weight != nullptr ? term.pair_weight[pair] : 1.0f) * term.pair_out[pair * dim + d];
    }
    return total;
}

// One block per output row r; src = rows ? rows[r] : r.
//   h = x[src] + sum_i gate_i[src] * scale_i * value_i[src];   if write_back: x[src] = h
//   out[r] = T(h * rsqrt(mean(h^2) + eps) * weight)            (out null: only the sum)
// All of it 32-bit.  It may be launched to start early, as the plain norm is: it waits for the kernel before it first of all.
constexpr int kTermThreads = 512;   // at most
template <typename T>
__global__ void __launch_bounds__(kTermThreads) residual_terms_kernel(float* __restrict__ x, const ResidualTerms terms, const float* __restrict__ weight, const int* __restrict__ rows,
                                      T* __restrict__ out, int dim, float eps, int write_back) {
    extern __shared__ __align__(16) float shared[];
    float* row_cache = shared;           // dim floats
    float* scratch = shared + (dim + 3) / 4 * 4;   // 33 floats
    wait_for_previous_kernel();
    allow_next_kernel();
    const int r = blockIdx.x;
    const size_t src = rows ? static_cast<size_t>(rows[r]) : static_cast<size_t>(r);
    float* xr = x + src * dim;
    float gate[kMaxTerms];
#pragma unroll
    for (int i = 0; i < kMaxTerms; ++i) gate[i] = i < terms.count && terms.term[i].gate != nullptr ? terms.term[i].gate[src * terms.term[i].gate_stride] : 1.0f;
    float sum = 0.0f;
    const bool four = dim % 4 == 0;
    if (four) {
        for (int d = 4 * threadIdx.x; d < dim; d += 4 * blockDim.x) {
            float4 h = *reinterpret_cast<const float4*>(xr + d);
#pragma unroll
            for (int i = 0; i < kMaxTerms; ++i) {
                if (i >= terms.count) break;
                const ResidualTerm& term = terms.term[i];
                const float4 v = term_value<T>(term, src, d, dim);
                const float4 s = term.scale != nullptr ? *reinterpret_cast<const float4*>(term.scale + d) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
                h.x += s.x * (gate[i] * v.x);
                h.y += s.y * (gate[i] * v.y);
                h.z += s.z * (gate[i] * v.z);
                h.w += s.w * (gate[i] * v.w);
            }
            if (write_back) *reinterpret_cast<float4*>(xr + d) = h;
            *reinterpret_cast<float4*>(row_cache + d) = h;
            sum += h.x * h.x + h.y * h.y + h.z * h.z + h.w * h.w;
        }
    } else {
        for (int d = threadIdx.x; d < dim; d += blockDim.x) {
            float h = xr[d];
            for (int i = 0; i < terms.count; ++i) {
                const ResidualTerm& term = terms.term[i];
                const float g = i == 0 ? gate[0] : i == 1 ? gate[1] : gate[2];
                h += (term.scale != nullptr ? term.scale[d] : 1.0f) * (g * term_value_one<T>(term, src, d, dim));
            }
            if (write_back) xr[d] = h;
            row_cache[d] = h;
            sum += h * h;
        }
    }
    if (out == nullptr) return;
    const float inv = rsqrtf(block_sum(sum, scratch) / static_cast<float>(dim) + eps);
    T* dst = out + static_cast<size_t>(r) * dim;
    if (four) {
        for (int d = 4 * threadIdx.x; d < dim; d += 4 * blockDim.x) {   // each thread rereads only what it wrote
            const float4 h = *reinterpret_cast<const float4*>(row_cache + d), w = *reinterpret_cast<const float4*>(weight + d);
            store_four(dst + d, make_float4(h.x * inv * w.x, h.y * inv * w.y, h.z * inv * w.z, h.w * inv * w.w));
        }
    } else {
        for (int d = threadIdx.x; d < dim; d += blockDim.x) dst[d] = from_float<T>(row_cache[d] * inv * weight[d]);
    }
}

}  // namespace lb

extern "C" {

// terms: `count` records on the host (see ResidualTerm); out null: only the sum (weight is not read then).  early 0: launched the ordinary
// way (where the stream has just waited for another stream).
int lb_residual_terms(float* x, const lb::ResidualTerm* terms, int count, const float* weight, const int* rows, void* out, int out_rows, int dim, float eps,
                      int write_back, int dtype, cudaStream_t stream, int early) {
    if (out_rows == 0) return 0;
    if (count < 0 || count > lb::kMaxTerms || dim < 1 || (out != nullptr && weight == nullptr)) return -2;
    lb::ResidualTerms all = {};
    all.count = count;
    for (int i = 0; i < count; ++i) {
        const lb::ResidualTerm& term = terms[i];
        const int kinds = (term.rows != nullptr) + (term.partials != nullptr) + (term.pair_out != nullptr);
        if (kinds != 1 || (term.partials != nullptr && (term.slices < 1 || (dim % 4 == 0 && term.slice_stride % 4 != 0))) ||
            (term.pair_out != nullptr && (term.top < 1 || term.pair_expert == nullptr)))
            return -2;
        all.term[i] = term;
    }
    const size_t shared = (static_cast<size_t>(dim) + 3 + 36) * sizeof(float);
    if (shared > 200 * 1024) return -2;
    // few rows: a thread per four elements, so that the kernel is one trip to memory long; many rows: more rows resident per SM
    int threads = dim >= 1024 ? 256 : 128;
    if (out_rows <= 64) {
        threads = ((dim + 3) / 4 + 31) / 32 * 32;
        threads = threads < 128 ? 128 : (threads > lb::kTermThreads ? lb::kTermThreads : threads);
    }
    LB_DISPATCH_DTYPE(dtype, {
        auto kernel = lb::residual_terms_kernel<T>;
        if (shared > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
        if (!early) kernel<<<out_rows, threads, shared, stream>>>(x, all, weight, rows, static_cast<T*>(out), dim, eps, write_back);
        else lb::launch_overlapped(kernel, dim3(out_rows), dim3(threads), shared, stream, x, all, weight, rows, static_cast<T*>(out), dim, eps, write_back);
    })
    return LB_LAUNCH_RESULT();
}

}  // extern "C"
