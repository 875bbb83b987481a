// Runs of tokens: recurrences of long prompts work on every run of C tokens of every sequence side by side. Run ci of
// sequence b is number q_start[b] / C + b + ci among all runs of the step: the numbers of different sequences do not meet,
// and there are at most T / C + B of them.
#pragma once
#include "common.cuh"

struct KbRun {
    int b, r0, n;               // the sequence, its first row of the run, the run's rows (0: no such run)
};
__device__ __forceinline__ KbRun kb_find_run(const int* __restrict__ q_start, int B, int C, int run) {
    int lo = 0, hi = B - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (q_start[mid] / C + mid <= run) lo = mid;
        else hi = mid - 1;
    }
    KbRun r;
    r.b = lo;
    const int ci = run - (q_start[lo] / C + lo);
    r.r0 = q_start[lo] + ci * C;
    r.n = max(0, min(C, q_start[lo + 1] - r.r0));
    return r;
}
