#include "recurrence.cuh"
namespace fa { namespace mixers {
int recurrence_segments(int, int, int, int, int, int, int, int* seg_len) { *seg_len = 1 << 30; return 1; }
bool recurrence_tc5_supported(const RecurrenceArgs&) { return false; }
cudaError_t launch_recurrence_tc5(const RecurrenceArgs&, cudaStream_t) { return cudaErrorNotSupported; }
} }
