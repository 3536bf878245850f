// Plain parameter structs shared by the kernels and the host launch API.
#pragma once

namespace sglb {

// Differential attention: query heads 2h and 2h + 1 are two soft-max maps over the same values; the head's output is
//   o = a_2h - lam * a_2h+1;   o / sqrt(mean(o^2) + eps) * post      (the mean over its dv values)
struct DiffCombine {
  float lam = 0.f, post = 1.f, eps = 0.f;
  int dv = 0;
};

}  // namespace sglb
