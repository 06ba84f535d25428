// model_base.hpp — what a ModelImpl needs besides its architecture: device allocations that die with the model, weight upload
// in the operand type, the bookkeeping of which tensors arrived, and seeded synthetic numbers.
#pragma once

#include <cmath>
#include <cstring>
#include <set>
#include <string>
#include <vector>

#include "../common.cuh"
#include "model.hpp"

namespace nvllm {

inline int pad8(int n) { return (n + 7) / 8 * 8; }

class ModelBase : public ModelImpl {
 public:
  ~ModelBase() override { for (void* p : allocs_) cudaFree(p); }
  bool weights_ready() const override { return ready_; }

 protected:
  ModelLimits lim_{};
  int dt_ = NVLLM_BF16;
  size_t esz_ = 2;
  std::set<std::string> needed_, loaded_;
  bool ready_ = false;

  template <typename T>
  int dalloc(T** p, size_t count, size_t elt = sizeof(T), bool zero = false) {
    void* q = nullptr;
    const size_t bytes = (count * elt + 255) & ~static_cast<size_t>(255);
    cudaError_t e = cudaMalloc(&q, bytes ? bytes : 256);
    if (e != cudaSuccess) { set_error("cudaMalloc of %zu bytes failed: %s", bytes, cudaGetErrorString(e)); return static_cast<int>(e); }
    allocs_.insert(q);
    if (zero) cudaMemset(q, 0, bytes ? bytes : 256);
    *p = static_cast<T*>(q);
    return 0;
  }
  int oalloc(void** p, size_t count, bool zero = false) { return dalloc(p, count, esz_, zero); }  // operand-typed buffer
  int valloc(float** p, size_t count, const std::string& name) { needed_.insert(name); return dalloc(p, count); }
  void release(void* p) { if (allocs_.erase(p)) cudaFree(p); }
  void* at(void* p, size_t elems) const { return static_cast<uint8_t*>(p) + elems * esz_; }   // operand-typed pointer arithmetic

  static float bf16_bits_to_f32(uint16_t b) {
    uint32_t u = static_cast<uint32_t>(b) << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
  }
  static uint16_t f32_to_bf16_bits(float f) {
    uint32_t u;
    memcpy(&u, &f, 4);
    return static_cast<uint16_t>((u + 0x7FFFu + ((u >> 16) & 1u)) >> 16);
  }
  // host bf16 values -> device operand tensor at ELEMENT offset `off`
  int put(void* dst, size_t off, const uint16_t* src, size_t n, cudaStream_t st) {
    const void* from = src;
    std::vector<float> tmp;
    if (esz_ == 4) {
      tmp.resize(n);
      for (size_t i = 0; i < n; ++i) tmp[i] = bf16_bits_to_f32(src[i]);
      from = tmp.data();
    }
    NVLLM_CUDA(cudaMemcpyAsync(at(dst, off), from, n * esz_, cudaMemcpyHostToDevice, st));
    NVLLM_CUDA(cudaStreamSynchronize(st));
    return 0;
  }
  // host bf16 [rows, cols] -> device f32, optionally transposed to [cols, rows]
  int putf(float* dst, const uint16_t* src, int64_t rows, int64_t cols, bool transpose, cudaStream_t st) {
    std::vector<float> tmp(static_cast<size_t>(rows) * cols);
    for (int64_t r = 0; r < rows; ++r)
      for (int64_t c = 0; c < cols; ++c) tmp[transpose ? c * rows + r : r * cols + c] = bf16_bits_to_f32(src[r * cols + c]);
    NVLLM_CUDA(cudaMemcpyAsync(dst, tmp.data(), tmp.size() * 4, cudaMemcpyHostToDevice, st));
    NVLLM_CUDA(cudaStreamSynchronize(st));
    return 0;
  }
  // counter-based standard-normal-like numbers: sum of four 16-bit uniforms
  static float gauss(uint64_t seed, uint64_t tensor, uint64_t i) {
    uint64_t x = seed ^ (tensor << 40) ^ (i + 1) * 0x9E3779B97F4A7C15ull;
    x ^= x >> 30; x *= 0xBF58476D1CE4E5B9ull;
    x ^= x >> 27; x *= 0x94D049BB133111EBull;
    x ^= x >> 31;
    const int s = static_cast<int>((x & 0xffff) + ((x >> 16) & 0xffff) + ((x >> 32) & 0xffff) + (x >> 48)) - 131070;
    return static_cast<float>(s) * 2.6428998e-05f;
  }
  static bool ends(const std::string& s, const char* suf) {
    const size_t n = strlen(suf);
    return s.size() >= n && s.compare(s.size() - n, n, suf) == 0;
  }

 private:
  std::set<void*> allocs_;
};

}  // namespace nvllm
