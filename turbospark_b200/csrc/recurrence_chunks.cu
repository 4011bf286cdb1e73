#include "recurrence_dev.cuh"
bool recurrence_chunks_supported(const Recurrence&) { return false; }
cudaError_t launch_recurrence_chunks(tsb_ctx*, cudaStream_t, const Recurrence&, const RowTiles&) { return cudaErrorNotSupported; }
