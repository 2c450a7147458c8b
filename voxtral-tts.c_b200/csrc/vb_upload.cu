/*
 * vb_upload.cu - the pinned staging ring of the weight uploads (vb_upload.cuh). The reference
 * copies every matrix with a blocking cudaMemcpy (voxtral_tts_cuda.cu:223-310).
 */
#include "vb_upload.cuh"

#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include <thread>
#include <vector>

namespace vb {

void Stager::open() {
    if (ok_) return;
    const char *env = getenv("VB200_UPLOAD_THREADS");
    unsigned hc = std::thread::hardware_concurrency();
    threads_ = env ? atoi(env) : (hc >= 4 ? 4 : 1);   /* four saturate the host's copy bandwidth where measured */
    if (threads_ < 1) threads_ = 1;
    if (threads_ > 32) threads_ = 32;
    for (int i = 0; i < kBufs; i++) {
        if (cudaHostAlloc(&pin_[i], cap_, cudaHostAllocDefault) != cudaSuccess ||
            cudaEventCreateWithFlags(&drained_[i], cudaEventDisableTiming) != cudaSuccess) {
            cudaGetLastError();
            return;   /* no pinned memory: copy() falls back to plain copies */
        }
        busy_[i] = false;
    }
    ok_ = true;
}

void Stager::close() {
    for (int i = 0; i < kBufs; i++) {
        if (pin_[i]) cudaFreeHost(pin_[i]);
        if (drained_[i]) cudaEventDestroy(drained_[i]);
        pin_[i] = nullptr; drained_[i] = nullptr; busy_[i] = false;
    }
    ok_ = false;
}

static void fill_parallel(char *dst, const char *src, size_t n, int threads) {
    const size_t min_part = (size_t)4 << 20;
    int parts = (int)((n + min_part - 1) / min_part);
    if (parts > threads) parts = threads;
    if (parts <= 1) { memcpy(dst, src, n); return; }
    const size_t per = ((n / parts) + 4095) & ~(size_t)4095;
    std::vector<std::thread> pool;
    for (int i = 1; i < parts; i++) {
        const size_t off = per * i;
        if (off >= n) break;
        const size_t len = off + per < n ? per : n - off;
        pool.emplace_back([=] { memcpy(dst + off, src + off, len); });
    }
    memcpy(dst, src, per < n ? per : n);
    for (auto &t : pool) t.join();
}

static int check(cudaError_t e, const char *what) {
    if (e == cudaSuccess) return 0;
    fprintf(stderr, "voxtral_b200: upload: %s failed: %s\n", what, cudaGetErrorString(e));
    return -1;
}

int Stager::copy(void *dst, const void *src, size_t bytes, cudaStream_t st) {
    bytes_copied += (double)bytes;
    if (!ok_) {
        if (check(cudaMemcpyAsync(dst, src, bytes, cudaMemcpyHostToDevice, st), "copy")) return -1;
        return check(cudaStreamSynchronize(st), "copy");
    }
    for (size_t off = 0; off < bytes; off += cap_) {
        const size_t n = bytes - off < cap_ ? bytes - off : cap_;
        const int b = next_;
        next_ = (next_ + 1) % kBufs;
        if (busy_[b] && check(cudaEventSynchronize(drained_[b]), "wait for a staging buffer")) return -1;
        fill_parallel((char *)pin_[b], (const char *)src + off, n, threads_);
        if (check(cudaMemcpyAsync((char *)dst + off, pin_[b], n, cudaMemcpyHostToDevice, st), "copy")) return -1;
        if (check(cudaEventRecord(drained_[b], st), "event")) return -1;
        busy_[b] = true;
    }
    return 0;
}

} // namespace vb
