// Which row of a table of biases a distance between two positions reads: a row per distance below half the rows, then rows
// whose reach grows geometrically up to the distance `most`; the last row serves everything beyond.
//   bucket(n) = n  for n < half,  else  min(rows - 1, half + floor(ln(n / half) / ln(most / half) * (rows - half))),  half = floor(rows / 2)
#pragma once
#include <algorithm>
#include <cmath>

namespace easygpt::host {

inline int distance_bucket(long long n, int rows, double most) {
    const int half = rows / 2;
    if (n < half) return (int)n;
    if (half == 0 || most <= (double)half) return rows - 1;       // no room for growing rows
    const double grown = std::log((double)n / half) / std::log(most / half) * (rows - half);
    // A distance that lies on a border exactly (n / half a power of the step) belongs to the upper row; the quotient of two
    // rounded logarithms may fall a few 1e-16 short of it.
    return (int)std::min<double>(rows - 1, half + std::floor(grown + 1e-11));
}

}  // namespace easygpt::host
