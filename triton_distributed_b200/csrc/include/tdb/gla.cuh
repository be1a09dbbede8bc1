// Shared pieces of the gated-linear-attention kernels (gla.cu, gla_chunk.cu).
#pragma once
#include "hybrid.h"
#include "ptx.cuh"

namespace tdb {

// log of sigmoid(z)^(1 / tau), stable for any z.
TDB_DEVICE float gla_log_decay(float z, float inv_tau) { return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau; }

}  // namespace tdb
