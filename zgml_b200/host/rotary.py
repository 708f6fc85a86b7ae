"""Frequency schedules of rotary positions, evaluated once at load: pair i of a head turns by position * f_i."""
import math

import numpy as np


def rotary_frequencies(rot: dict) -> np.ndarray:
    """[dims / 2] f32, f_i = base^(-2i / dims), slowed as `scaling` says:
      * {"factor"}: every pair turns `factor` times slower (linear scaling);
      * {"factor", "low", "high", "original"}: a pair whose wavelength 2 pi / f is shorter than original / high keeps f, one longer
        than original / low turns `factor` times slower, and in between the two are blended linearly in original / wavelength."""
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    sc = rot.get("scaling")
    if sc and "original" in sc:
        factor, low, high, original = float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"])
        wl = 2.0 * math.pi / f
        blend = (original / wl - low) / (high - low) if high != low else np.ones_like(f)
        mixed = (1.0 - blend) * f / factor + blend * f
        f = np.where(wl < original / high, f, np.where(wl > original / low, f / factor, mixed))
    elif sc:
        f = f / float(sc["factor"])
    return f.astype(np.float32)
