#include "float_common.cuh"
namespace zkds {
bool scan_tc_takes(const zkfp_scan_args&) { return false; }
int launch_scan_tc(const zkfp_scan_args&, cudaStream_t) { return ZKDS_ERR_UNSUPPORTED; }
long long scan_tc_scratch(const zkfp_scan_args&) { return 0; }
}
