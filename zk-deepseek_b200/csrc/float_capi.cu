// extern "C" surface of libfloatops.so: argument checks, kernel choice, launch accounting (include/zkds_float.h).
#include <atomic>

#include "float_common.cuh"

namespace zkds {

static thread_local int t_cuda_error = 0;
static std::atomic<long long> g_launches{0};

int set_cuda_error(cudaError_t e)
{
    if (e == cudaSuccess) return ZKDS_OK;
    t_cuda_error = (int)e;
    return ZKDS_ERR_CUDA;
}

int check_launch() { return set_cuda_error(cudaGetLastError()); }

int fp_launched()
{
    g_launches.fetch_add(1, std::memory_order_relaxed);
    return check_launch();
}

int fp_sm_count()
{
    static int sms[64];
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
    if (!sms[dev]) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
        sms[dev] = n;
    }
    return sms[dev];
}

static int* g_flag_host[64];
static int* g_flag_dev[64];

int* fp_error_flag()
{
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
    if (!g_flag_host[dev]) {
        int* h = nullptr;
        if (cudaHostAlloc((void**)&h, 64, cudaHostAllocMapped) != cudaSuccess) return nullptr;
        h[0] = 0;
        int* d = nullptr;
        if (cudaHostGetDevicePointer((void**)&d, h, 0) != cudaSuccess) return nullptr;
        g_flag_dev[dev] = d;
        g_flag_host[dev] = h;
    }
    return g_flag_dev[dev];
}

// up to here a linear layer streams its weights through the CUDA cores
static constexpr long long kStreamRowsBf16 = 2, kStreamRowsF32 = 16;

static bool linear_ok(const zkfp_linear_args* a)
{
    if (!a || !a->A || !a->W || !a->out || a->M < 0 || a->N <= 0 || a->K <= 0) return false;
    if ((a->N & 7) || (a->K & 7) || (a->lda & 7) || (a->ldw & 7) || (a->ldo & 7)) return false;
    if (a->lda < a->K || a->ldw < a->K || a->M > 0x7fffffffll || a->N > 0x7fffffffll || a->K > 0x7fffffffll) return false;
    if ((uintptr_t)a->A & 15 || (uintptr_t)a->W & 15 || (uintptr_t)a->out & 15) return false;
    if (a->out2 && (a->epilogue == ZKFP_EPI_GLU || a->epilogue == ZKFP_EPI_GATE || a->split <= 0 || a->split >= a->N || (a->split & 31) ||
                    a->ldo2 < a->N - a->split || (a->ldo2 & 7) || ((uintptr_t)a->out2 & 15)))
        return false;
    if ((uintptr_t)a->bias & 15) return false;
    if (a->epilogue != ZKFP_EPI_GLU && a->ldo < (a->out2 ? a->split : a->N)) return false;
    if (a->epilogue == ZKFP_EPI_GLU && ((a->N & 15) || a->ldo < a->N / 2)) return false;
    if (a->epilogue == ZKFP_EPI_ROTATE &&
        (!a->table || !a->start || a->seq <= 0 || a->positions <= 0 || a->positions > 0x7fffffffll || a->period <= 0 || (a->period & 1) || (a->offset & 1) ||
         a->rot_begin < 0 || (a->rot_begin & 1) || (a->rot_end & 1) || a->rot_end > a->N))
        return false;
    if (a->epilogue == ZKFP_EPI_GATE && (!a->aux || (a->ldaux & 7) || ((uintptr_t)a->aux & 15))) return false;
    return a->epilogue >= 0 && a->epilogue <= ZKFP_EPI_GLU && (a->dtype | a->out_dtype) <= 1;
}

static bool attention_ok(const zkfp_attention_args* a)
{
    return a && a->q && a->k1 && a->k2 && a->v && a->out && a->start && a->batch > 0 && a->batch < 65536 && a->seq >= 0 &&
           a->heads > 0 && a->heads < 65536 && a->d1 > 0 && a->d2 >= 0 && a->dv > 0 && !(a->d1 & 7) && !(a->d2 & 7) &&
           !(a->dv & 7) && a->q_head >= a->d1 + a->d2 && a->o_head >= a->dv && (a->shared || a->batch == 1) && a->heads_per_kv >= 0 &&
           (a->heads_per_kv <= 1 || (!a->shared && a->heads % a->heads_per_kv == 0)) &&
           (!a->gate || (!a->shared && !((a->gate_tok | a->gate_head) & 7) && !((uintptr_t)a->gate & 15))) &&
           (!a->o_tok || (!a->shared && a->o_tok >= a->heads * a->o_head && !(a->o_tok & 7)));
}

}  // namespace zkds

using namespace zkds;

extern "C" {

int zkfp_linear_path(const zkfp_linear_args* a)
{
    if (a->M <= (a->dtype == ZKFP_BF16 ? kStreamRowsBf16 : kStreamRowsF32)) return 2;
    return a->dtype == ZKFP_BF16 ? 1 : 0;
}

int zkfp_linear(const zkfp_linear_args* a, void* stream)
{
    if (!linear_ok(a)) return ZKDS_ERR_ARG;
    if (a->M == 0) return ZKDS_OK;
    LinEpi e;
    e.out = a->out; e.aux = a->aux; e.table = (const float2*)a->table; e.start = a->start;
    e.ldo = a->ldo; e.ldaux = a->ldaux; e.seq = a->seq > 0 ? a->seq : 1; e.positions = a->positions;
    e.kind = a->epilogue; e.out_bf16 = a->out_dtype; e.aux_bf16 = a->dtype;
    e.pairs = a->pairs; e.period = a->period > 0 ? a->period : 1; e.offset = a->offset;
    e.rot_begin = a->rot_begin; e.rot_end = a->rot_end > 0 ? a->rot_end : (int)a->N;
    e.bias = a->bias; e.out2 = a->out2; e.ldo2 = a->ldo2; e.split = a->out2 ? a->split : a->N;
    cudaStream_t st = (cudaStream_t)stream;
    switch (zkfp_linear_path(a)) {
    case 2: return launch_linear_stream(*a, e, st);
    case 1: return launch_linear_tc(*a, e, st);
    default: return launch_linear_plain(*a, e, st);
    }
}

int zkfp_attention_path(const zkfp_attention_args* a)
{
    if (a->dtype != ZKFP_BF16) return 0;
    return (a->shared ? attention_decode_tc_takes(*a) : attention_prefill_tc_takes(*a)) ? 1 : 0;
}

long long zkfp_attention_scratch(const zkfp_attention_args* a)
{
    return a->shared && zkfp_attention_path(a) == 1 ? attention_decode_scratch(*a) : 0;
}

int zkfp_attention(const zkfp_attention_args* a, void* stream)
{
    if (!attention_ok(a)) return ZKDS_ERR_ARG;
    if (a->seq == 0) return ZKDS_OK;
    cudaStream_t st = (cudaStream_t)stream;
    if (zkfp_attention_path(a) == 1)
        return a->shared ? launch_attention_decode_tc(*a, st) : launch_attention_prefill_tc(*a, st);
    return launch_attention_plain(*a, st);
}

int zkfp_device_status(void)
{
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64 || !g_flag_host[dev]) return ZKDS_OK;
    volatile int* h = g_flag_host[dev];
    const int v = h[0];
    h[0] = 0;
    return v ? ZKDS_ERR_DEVICE : ZKDS_OK;
}

long long zkfp_launches(void) { return g_launches.load(); }
int zkfp_cuda_error(void) { return t_cuda_error; }

}  // extern "C"
