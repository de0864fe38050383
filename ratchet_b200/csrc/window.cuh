// Arguments of the windowed-attention kernels (latent_attention.cu, window_tc.cu).
#pragma once
#include "common.cuh"

struct WindowArgs {
    const void *q, *kv, *shared;
    void* out;
    long long shared_pitch;
    int T, L, H, D, R, E, window;     // D: own key features of a head, R: shared ones (a query has D + R)
    float scale;
};

// RCU_ERR_UNSUPPORTED: sizes or alignments the tensor maps do not take
rcu_status rcu_window_tc(rcu_device* dev, const WindowArgs& a);
