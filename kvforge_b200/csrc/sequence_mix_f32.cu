// The kernels of sequence_mix.cuh for float storage (a translation unit per storage type: they compile side by side).
#include "sequence_mix.cuh"

KVF_SEQMIX_API(f32, float)

// Turn programmatic dependent launch on or off for every launch of this library (the flag is one per shared library).
KVF_API int kvf_mixers_set_pdl(int enabled) {
  kvf::g_pdl_enabled = enabled ? 1 : 0;
  return 0;
}
