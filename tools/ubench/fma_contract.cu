// fma_contract.cu -- which product of a*b - c*d and of a*b + c*d does nvcc fuse when contraction is on (its default)?
// Three kernels evaluate the two rotary expressions as they are written in the source; the host compares every output
// with the three candidates (no product fused, the first, the second) and counts the differences.  The reference-order
// kernels and the CPU oracle spell the placement that this reports (the one with no difference) with explicit fmas:
// the first product of the sum as written is fused.
//   nvcc -gencode arch=compute_100a,code=sm_100a -O3 -o fma_contract fma_contract.cu && ./fma_contract
#include <cmath>
#include <cstdint>
#include <cstdio>
#include <vector>
#include <cuda_runtime.h>

__global__ void rot(const float* x0, const float* x1, const float* c, const float* s, float* v1, float* v2, float* sq, int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  v1[i] = x0[i] * c[i] - x1[i] * s[i];
  v2[i] = x1[i] * c[i] + x0[i] * s[i];
  float sum = x0[i];
  sum += x1[i] * x1[i];
  sq[i] = sum;
}

int main() {
  const int n = 1 << 20;
  std::vector<float> h[7];
  uint64_t z = 88172645463325252ull;
  for (int k = 0; k < 7; ++k) {
    h[k].resize(n);
    for (int i = 0; i < n && k < 4; ++i) {
      z ^= z << 13, z ^= z >> 7, z ^= z << 17;
      h[k][i] = (float)((double)(z >> 11) / 9007199254740992.0 * 2.0 - 1.0);
    }
  }
  float* d[7];
  for (int k = 0; k < 7; ++k) {
    if (cudaMalloc(&d[k], n * sizeof(float)) != cudaSuccess) return 1;
    cudaMemcpy(d[k], h[k].data(), n * sizeof(float), cudaMemcpyHostToDevice);
  }
  rot<<<n / 256, 256>>>(d[0], d[1], d[2], d[3], d[4], d[5], d[6], n);
  for (int k = 4; k < 7; ++k) cudaMemcpy(h[k].data(), d[k], n * sizeof(float), cudaMemcpyDeviceToHost);
  if (cudaDeviceSynchronize() != cudaSuccess) return 1;
  long diff[3][3] = {};
  for (int i = 0; i < n; ++i) {
    const float a = h[0][i], b = h[1][i], c = h[2][i], s = h[3][i];
    volatile float ac = a * c, bs = b * s, as = a * s, bc = b * c, bb = b * b;
    const float w1[3] = {ac - bs, fmaf(a, c, -bs), fmaf(-b, s, ac)};
    const float w2[3] = {bc + as, fmaf(b, c, as), fmaf(a, s, bc)};
    const float w3[3] = {a + bb, fmaf(b, b, a), fmaf(b, b, a)};
    for (int k = 0; k < 3; ++k) diff[0][k] += h[4][i] != w1[k], diff[1][k] += h[5][i] != w2[k], diff[2][k] += h[6][i] != w3[k];
  }
  const char* e[3] = {"x0*c - x1*s", "x1*c + x0*s", "sum += x*x"};
  for (int k = 0; k < 3; ++k) printf("%s: differences from none fused %ld, first product fused %ld, second fused %ld of %d\n", e[k], diff[k][0], diff[k][1], diff[k][2], n);
  return 0;
}
