// Activations of two operands alone (csrc/gates.cuh), for the products whose epilogue does not take them.
// Compiled without fast math.
#include "common.cuh"
#include "gates.cuh"

namespace tyr {

struct GateArgs {
  const void* z;               // [rows, ldz]
  const void* e;               // [rows, lde]: the second operand; null: z holds, per 2 * block columns, `block` gate columns and their up columns
  void* out;                   // [rows, n]
  long long ldz, lde, rows;
  int n, block, kind;          // 8: clamped SwiGLU (a: limit, b: slope), 9: tanh-GELU of z times e
  float a, b;
};

template <typename T>
__global__ void __launch_bounds__(256) gates_kernel(GateArgs a) {
  pdl_entry();
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < a.rows * a.n; i += gridDim.x * 256LL) {
    const long long row = i / a.n;
    const int c = static_cast<int>(i % a.n);
    const T* z = static_cast<const T*>(a.z) + row * a.ldz;
    float v;
    if (a.kind == 8) {
      const int g = c / a.block * 2 * a.block + c % a.block;
      v = clamped_swiglu(static_cast<float>(z[g]), static_cast<float>(z[g + a.block]), a.a, a.b);
    } else {
      v = gelu_tanh(static_cast<float>(z[c])) * static_cast<float>(static_cast<const T*>(a.e)[row * a.lde + c]);
    }
    static_cast<T*>(a.out)[i] = static_cast<T>(v);
  }
}

}  // namespace tyr

using namespace tyr;

static int gates_launch(const GateArgs& a, int dtype, void* stream) {
  if (a.rows <= 0 || a.n <= 0 || a.block <= 0) return -1;
  const long long want = (a.rows * a.n + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  return (int)(dtype == 1 ? launch_dependent(gates_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, a)
                          : launch_dependent(gates_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, a));
}

// out [rows, n] = clamped SwiGLU of z [rows, >= 2 n], whose columns are blocks of `block` gate columns and the matching up columns.
extern "C" TYR_EXPORT int tyr_clamped_swiglu(const void* z, long long ldz, void* out, long long rows, int n, int block, float limit, float slope,
                                             int dtype, void* stream) {
  return gates_launch(GateArgs{z, nullptr, out, ldz, 0, rows, n, block, 8, limit, slope}, dtype, stream);
}

// out [rows, n] = gelu(z) * e (tanh form).
extern "C" TYR_EXPORT int tyr_gelu_mul(const void* z, long long ldz, const void* e, long long lde, void* out, long long rows, int n, int dtype,
                                       void* stream) {
  if (e == nullptr) return -1;
  return gates_launch(GateArgs{z, e, out, ldz, lde, rows, n, 1, 9, 0.f, 0.f}, dtype, stream);
}
