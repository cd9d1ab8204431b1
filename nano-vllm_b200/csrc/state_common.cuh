// What the matrix-state kernels share: the gates of scalar linear attention, and the tensor-core form's entry.
#pragma once
#include "mix_common.cuh"

__device__ __forceinline__ float softplus_(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// What scalar linear attention does with a token: raw fp32 (or T) inputs -> (log decay, write weight).
template <typename T>
struct ScalarGate {
    const T* raw;             // step-size pre-activations (n, >= H), or NULL: `log_decay` and `write` are given
    const float *log_decay, *write;
    int64_t stride;           // of whichever is read
    const float *rate, *bias;
    __device__ __forceinline__ float2 fetch(int64_t row, int h) const {      // loads only
        if (raw) return make_float2(ldf(raw + row * stride + h), 0.f);
        return make_float2(log_decay[row * stride + h], write[row * stride + h]);
    }
    __device__ __forceinline__ float2 gates(float2 f, float rt, float b) const {
        if (!raw) return f;
        const float dt = softplus_(f.x + b);
        return make_float2(rt * dt, dt);
    }
};

// Prompt portions of scalar linear attention on the tensor cores (chunk_state.cu).  Returns B200_EUNSUPPORTED for shapes and alignments it does
// not take; the caller then runs the fp32-pipe form.  Arguments as for b200m_linear_state.
int chunk_state_launch(const __nv_bfloat16* x, int64_t stride, int q_off, int k_off, int v_off, const ScalarGate<__nv_bfloat16>& sg, float* state,
                       const int32_t* state_slots, const int32_t* cu_q, const int32_t* cu_k, float* out, int num_seqs, int H, int G, int dim,
                       int vdim, int ones, float q_scale, cudaStream_t st);
