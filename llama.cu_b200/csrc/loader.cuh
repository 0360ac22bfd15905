// File -> device loader shared by the model families.
#pragma once
#include <fcntl.h>
#include <sys/stat.h>
#include <unistd.h>

#include <algorithm>
#include <atomic>
#include <string>
#include <thread>
#include <vector>

#include "runtime.cuh"

namespace lcu {

// Staged loader: files are read in pieces into two pinned buffers; while one piece travels to the device
// (cudaMemcpyAsync on the loader's stream, one copy per piece) the next one is read from the file.  One loader per
// GPU of the partition; finish() waits for the last copies.
struct staged_loader {
  static constexpr size_t PIECE = (size_t)64 << 20;
  static constexpr int READERS = 8;
  int device = 0;
  void* pin[2] = {nullptr, nullptr};
  cudaEvent_t done[2] = {nullptr, nullptr};
  bool in_flight[2] = {false, false};
  cudaStream_t stream = nullptr;
  int cur = 0;

  int init(int dev) {
    device = dev;
    device_guard g(dev);
    LCU_CUDA(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking));
    for (int i = 0; i < 2; ++i) {
      LCU_CUDA(cudaMallocHost(&pin[i], PIECE));
      LCU_CUDA(cudaEventCreateWithFlags(&done[i], cudaEventDisableTiming));
    }
    return LCU_OK;
  }
  ~staged_loader() {
    device_guard g(device);
    if (stream) cudaStreamSynchronize(stream);
    for (int i = 0; i < 2; ++i) {
      if (pin[i]) cudaFreeHost(pin[i]);
      if (done[i]) cudaEventDestroy(done[i]);
    }
    if (stream) cudaStreamDestroy(stream);
  }
  int copy_file(const std::string& path, void* dst, size_t bytes, size_t file_off, size_t file_bytes) {
    int fd = open(path.c_str(), O_RDONLY);
    if (fd < 0) {
      set_last_error("cannot open %s", path.c_str());
      return LCU_ERR_IO;
    }
    struct stat st;
    if (fstat(fd, &st) != 0 || (size_t)st.st_size != file_bytes) {
      close(fd);
      set_last_error("%s: expected %zu bytes, file has %lld", path.c_str(), file_bytes, (long long)st.st_size);
      return LCU_ERR_IO;
    }
#ifdef POSIX_FADV_SEQUENTIAL
    posix_fadvise(fd, 0, 0, POSIX_FADV_SEQUENTIAL);
#endif
    device_guard g(device);
    for (size_t off = 0; off < bytes;) {
      const size_t n = std::min(PIECE, bytes - off);
      if (in_flight[cur]) {  // the buffer's previous piece must have left it
        if (cudaEventSynchronize(done[cur]) != cudaSuccess) {
          close(fd);
          set_last_error("copy of %s to the device failed", path.c_str());
          return LCU_ERR_CUDA;
        }
        in_flight[cur] = false;
      }
      // the piece is read by several threads at once (a single reader copies out of the page cache at a fraction of
      // what the host-to-device link takes)
      const int n_readers = n >= ((size_t)4 << 20) ? READERS : 1;
      const size_t share = (n / n_readers + 4095) & ~(size_t)4095;
      std::atomic<int> failed{0};
      auto read_range = [&](size_t lo, size_t hi) {
        while (lo < hi) {
          const ssize_t r = pread(fd, (char*)pin[cur] + lo, hi - lo, (off_t)(file_off + off + lo));
          if (r <= 0) {
            failed = 1;
            return;
          }
          lo += (size_t)r;
        }
      };
      std::vector<std::thread> readers;
      for (int t = 1; t < n_readers; ++t) readers.emplace_back(read_range, std::min(n, t * share), std::min(n, (t + 1) * share));
      read_range(0, std::min(n, share));
      for (auto& th : readers) th.join();
      if (failed) {
        close(fd);
        set_last_error("short read from %s", path.c_str());
        return LCU_ERR_IO;
      }
      cudaError_t e = cudaMemcpyAsync((char*)dst + off, pin[cur], n, cudaMemcpyHostToDevice, stream);
      if (e == cudaSuccess) e = cudaEventRecord(done[cur], stream);
      if (e != cudaSuccess) {
        close(fd);
        set_last_error("copy of %s to the device failed: %s", path.c_str(), cudaGetErrorString(e));
        return LCU_ERR_CUDA;
      }
      in_flight[cur] = true;
      cur ^= 1;
      off += n;
    }
    close(fd);
    return LCU_OK;
  }
  int finish() {
    device_guard g(device);
    LCU_CUDA(cudaStreamSynchronize(stream));
    in_flight[0] = in_flight[1] = false;
    return LCU_OK;
  }
};

}  // namespace lcu
