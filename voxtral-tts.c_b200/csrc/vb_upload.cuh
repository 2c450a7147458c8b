/*
 * vb_upload.cuh - host -> device copies of model weights through a ring of pinned staging
 * buffers, shared by every model the library loads.
 *
 * A few host threads fill buffer n + 1 from the caller's (pageable, usually memory-mapped) memory
 * while the copy engine drains buffer n; repacking kernels run behind the copies on the same
 * stream. Nothing waits for the device except a buffer that is still being drained; the upload
 * call synchronises once at its end.
 */
#ifndef VB_UPLOAD_CUH
#define VB_UPLOAD_CUH

#include <cuda_runtime.h>
#include <stddef.h>

namespace vb {

class Stager {
public:
    /* Pins the ring (VB200_UPLOAD_THREADS host threads fill it). Without pinned memory copy() falls
     * back to plain blocking copies. */
    void open();
    void close();
    /* Asynchronous on `st` as far as the device goes; the source may be reused on return. */
    int copy(void *dst, const void *src, size_t bytes, cudaStream_t st);
    double bytes_copied = 0.0;

private:
    static const int kBufs = 3;
    size_t cap_ = (size_t)64 << 20;
    void *pin_[kBufs] = {};
    cudaEvent_t drained_[kBufs] = {};
    bool busy_[kBufs] = {};
    int next_ = 0, threads_ = 4;
    bool ok_ = false;
};

} // namespace vb

#endif
