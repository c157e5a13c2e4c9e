// Number of kernels of this extension launched since the last reset (all threads).
#include <atomic>

static std::atomic<long long> g_launches{0};
extern "C" void rb_note_launch(int n) { g_launches.fetch_add(n, std::memory_order_relaxed); }
extern "C" long long rb_launch_count() { return g_launches.load(std::memory_order_relaxed); }
extern "C" void rb_reset_launch_count() { g_launches.store(0, std::memory_order_relaxed); }
