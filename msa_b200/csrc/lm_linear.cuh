// Argument checks shared by the two files of the recurrences.
#pragma once
#include "lm_common.cuh"

namespace msa {
int wkv_check(const msa_lm_wkv_args* a, const char* what);
int ssd_check(const msa_lm_ssd_args* a, const char* what);
}  // namespace msa
