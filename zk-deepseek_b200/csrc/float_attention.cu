#include "float_common.cuh"
namespace zkds {
bool attention_prefill_tc_takes(const zkfp_attention_args&) { return false; }
int launch_attention_prefill_tc(const zkfp_attention_args& a, cudaStream_t st) { return launch_attention_plain(a, st); }
bool attention_decode_tc_takes(const zkfp_attention_args&) { return false; }
int launch_attention_decode_tc(const zkfp_attention_args& a, cudaStream_t st) { return launch_attention_plain(a, st); }
long long attention_decode_scratch(const zkfp_attention_args&) { return 0; }
}
