// Arguments of the masked-attention kernels of prompts (latent_attention.cu, window_tc.cu): rows of keys and values that every query
// sees a run of, ending with itself.
#pragma once
#include "common.cuh"

// Where a query's run of visible rows begins, in rows of the keys: rows are consecutive positions, `position` that of row 0.
struct Visible {
    int window;               // sliding: the query and the window - 1 rows before it
    int chunk;                // > 0 instead: the rows in the same run of `chunk` positions
    uint32_t position;
    __host__ __device__ __forceinline__ int first(int row) const {
        const int lo = chunk > 0 ? row - (int)((position + (uint32_t)row) % (uint32_t)chunk) : row - window + 1;
        return lo > 0 ? lo : 0;
    }
};

struct WindowArgs {
    const void *q, *kv, *shared;      // kv rows: G heads' keys of D features, then G heads' values of E
    void* out;
    long long shared_pitch;
    int T, L, H, G, D, R, E;          // D: own key features of a head, R: features shared by the heads (a query has D + R)
    Visible see;
    float scale;
    const float* sink;                // [H], nullable: exp(sink) joins the softmax denominator
};

// The kernel for the sizes and type at hand (latent_attention.cu)
rcu_status rcu_attend(rcu_device* dev, int dt, const WindowArgs& a);
// bf16 blocks on tcgen05; RCU_ERR_UNSUPPORTED: sizes or alignments the tensor maps do not take (window_tc.cu)
rcu_status rcu_window_tc(rcu_device* dev, const WindowArgs& a);
