// Differential attention: a head's two softmax maps a and b over the same values become
//     o = a - lam b,   y = o / sqrt(sum(o^2) / vdim + eps) * gain,
// lam, eps and gain one number each, the sum over the head's `vdim` true elements; float32 until y is stored.
#pragma once
struct PairOut {
    int on;                      // 0: heads stay as they are
    float lam, eps, gain;
    int vdim, width;             // true elements of a head, elements of a stored row (zeros behind the true ones)
};
