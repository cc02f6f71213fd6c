"""Rotary position tables: angle frequencies, their YaRN interpolation, and the (cos, sin) table the kernels read.

Everything is computed in double precision here and stored as float32, so that a kernel never evaluates an angle: at a
distant position the product position * frequency would otherwise lose more bits than the table entry holds.
"""
import math

import numpy as np


def frequencies(dims, base):
    """base^(-2 i / dims) for the dims / 2 rotated pairs."""
    return float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)


def yarn(freq, dims, base, factor, original, fast, slow):
    """YaRN: pairs that turn more than `fast` times within the original context keep their frequency, those that turn less
    than `slow` times have it divided by `factor`, those between are blended by a ramp over the pair index. Returns
    (frequencies, amplitude of cos and sin)."""
    def pair_of(turns):
        return dims * math.log(original / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(fast)), 0)
    hi = min(math.ceil(pair_of(slow)), dims - 1)
    ramp = np.clip((np.arange(dims // 2, dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq * (1.0 - ramp) + freq / factor * ramp, 0.1 * math.log(factor) + 1.0


def rotary_table(max_len, dims, base, scaling=None):
    """float32 [max_len, dims / 2, 2]: (cos, sin) of position * frequency, amplitude included. `scaling`: the arguments of
    `yarn` after the base, as a dict."""
    freq, amp = frequencies(dims, base), 1.0
    if scaling:
        freq, amp = yarn(freq, dims, base, **scaling)
    ang = np.arange(max_len, dtype=np.float64)[:, None] * freq[None, :]
    return np.stack([np.cos(ang) * amp, np.sin(ang) * amp], axis=-1).astype(np.float32)
