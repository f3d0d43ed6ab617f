// Argument checks shared by the extern "C" entry points of both libraries.
#pragma once
#include "common.cuh"

namespace sk {

static inline bool aligned(const void* p, size_t a) { return (reinterpret_cast<uintptr_t>(p) % a) == 0; }
static inline bool valid_dtype(int d) { return d == SK_F32 || d == SK_BF16 || d == SK_F16; }
static inline size_t esize(int d) { return d == SK_F32 ? 4 : 2; }
static inline size_t up256(size_t x) { return (x + 255) & ~(size_t)255; }

}  // namespace sk

#define SK_REQUIRE(cond, ...)                                          \
    do {                                                               \
        if (!(cond)) return fail(SK_ERR_INVALID_ARGUMENT, __VA_ARGS__); \
    } while (0)
#define SK_ALIGNED(ptr, a, name)                                                         \
    do {                                                                                 \
        if (!aligned(ptr, a)) return fail(SK_ERR_MISALIGNED, name " must be %d-byte aligned", (int)(a)); \
    } while (0)
