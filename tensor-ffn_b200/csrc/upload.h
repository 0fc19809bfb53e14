// Host-to-device helpers of the weight loaders and sessions.
#pragma once
#include "engine.h"
#include <algorithm>
#include <cstring>

namespace tffn {

inline void upload(DeviceBuffer& dst, const void* src, size_t bytes) {
    dst.alloc(bytes);
    TFFN_CUDA(cudaMemcpy(dst.p, src, bytes, cudaMemcpyHostToDevice));
    // from pageable memory the call may return once the data is staged: wait for it to reach the device,
    // the streams that will read it are not ordered after the default stream
    TFFN_CUDA(cudaStreamSynchronize(0));
}

// Host-to-device staging for the loaders: the weight files are memory-mapped (pageable), so a plain
// cudaMemcpy would page each tensor in, stage it inside the driver and block. Here the host thread copies the
// next chunk out of the mapping into one of two pinned buffers while the copy engine still moves the previous
// one; everything (copies, the re-layout kernels that follow them) is ordered on one stream and the loader
// waits once at the end.
class Stager {
public:
    explicit Stager(size_t chunk_bytes = (size_t)32 << 20) : chunk_(chunk_bytes) {
        TFFN_CUDA(cudaStreamCreateWithFlags(&s_, cudaStreamNonBlocking));
        for (int i = 0; i < 2; ++i) {
            TFFN_CUDA(cudaMallocHost((void**)&buf_[i], chunk_));
            TFFN_CUDA(cudaEventCreateWithFlags(&ev_[i], cudaEventDisableTiming));
        }
    }
    ~Stager() {
        cudaStreamSynchronize(s_);
        for (int i = 0; i < 2; ++i) {
            if (buf_[i]) cudaFreeHost(buf_[i]);
            if (ev_[i]) cudaEventDestroy(ev_[i]);
        }
        cudaStreamDestroy(s_);
    }
    Stager(const Stager&) = delete;
    Stager& operator=(const Stager&) = delete;
    cudaStream_t stream() const { return s_; }
    void copy(void* dst, const void* src, size_t bytes) {
        for (size_t o = 0; o < bytes; o += chunk_) put((char*)dst + o, (const char*)src + o, std::min(chunk_, bytes - o), 0, 0, 0);
    }
    // `rows` rows of `width` bytes, `src_pitch` bytes apart in the mapping -> dense on the device
    void copy2d(void* dst, const void* src, size_t src_pitch, size_t width, size_t rows) {
        if (width == 0 || rows == 0) return;
        if (src_pitch == width) return copy(dst, src, width * rows);
        if (width > chunk_) throw Error(kErrUnsupported, "a matrix row is longer than the staging buffer");
        const size_t rows_per = chunk_ / width;
        for (size_t r = 0; r < rows; r += rows_per) {
            const size_t nr = std::min(rows_per, rows - r);
            put((char*)dst + r * width, (const char*)src + r * src_pitch, nr * width, src_pitch, width, nr);
        }
    }
    void finish() { TFFN_CUDA(cudaStreamSynchronize(s_)); }

private:
    // one chunk: wait until the pinned buffer's previous transfer has left it, fill it, send it
    void put(void* dst, const char* src, size_t bytes, size_t pitch, size_t width, size_t rows) {
        uint8_t* b = buf_[cur_];
        if (used_[cur_]) TFFN_CUDA(cudaEventSynchronize(ev_[cur_]));
        if (rows == 0) {
            memcpy(b, src, bytes);
        } else {
            for (size_t r = 0; r < rows; ++r) memcpy(b + r * width, src + r * pitch, width);
        }
        TFFN_CUDA(cudaMemcpyAsync(dst, b, bytes, cudaMemcpyHostToDevice, s_));
        TFFN_CUDA(cudaEventRecord(ev_[cur_], s_));
        used_[cur_] = true;
        cur_ ^= 1;
    }
    size_t chunk_;
    cudaStream_t s_ = nullptr;
    uint8_t* buf_[2] = {nullptr, nullptr};
    cudaEvent_t ev_[2] = {nullptr, nullptr};
    bool used_[2] = {false, false};
    int cur_ = 0;
};

// carves 256-byte aligned views out of one allocation
struct Slab {
    DeviceBuffer* mem;
    size_t off = 0;
    void take(DeviceBuffer& dst, size_t bytes) {
        const size_t a = (off + 255) & ~(size_t)255;
        if (a + bytes > mem->bytes) throw Error(kErrInvalid, "weight slab too small (internal size computation)");
        dst.view((char*)mem->p + a, bytes);
        off = a + bytes;
    }
    static size_t padded(size_t bytes) { return (bytes + 255) & ~(size_t)255; }
};

}  // namespace tffn
