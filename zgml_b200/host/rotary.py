"""Frequency schedules of rotary positions, evaluated once at load: pair i of a head turns by position * f_i."""
import math

import numpy as np


def rotary_frequencies(rot: dict) -> np.ndarray:
    """[dims / 2] f32, f_i = base^(-2i / dims), slowed as `scaling` says:
      * {"factor"}: every pair turns `factor` times slower (linear scaling);
      * {"factor", "fast", "slow", "original"} (YaRN, Peng et al., "YaRN: Efficient Context Window Extension of Large Language Models"): pairs that turn
        more than `fast` times over the original context keep f, pairs that turn less than `slow` times turn `factor` times slower, with
        a linear ramp over the pair's index in between; `rotary_magnitude` is what cosines and sines are multiplied by;
      * {"factor", "low", "high", "original"}: a pair whose wavelength 2 pi / f is shorter than original / high keeps f, one longer
        than original / low turns `factor` times slower, and in between the two are blended linearly in original / wavelength."""
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    sc = rot.get("scaling")
    if sc and "fast" in sc:
        factor, original, ln_base = float(sc["factor"]), float(sc["original"]), math.log(float(rot["base"]))

        def index_of(turns):       # the (fractional) pair that turns `turns` times over the original context
            return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * ln_base)

        lo, hi = max(math.floor(index_of(float(sc["fast"]))), 0), min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
        ramp = np.clip((np.arange(dims // 2, dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        f = f / factor * ramp + f * (1.0 - ramp)
    elif sc and "original" in sc:
        factor, low, high, original = float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"])
        wl = 2.0 * math.pi / f
        blend = (original / wl - low) / (high - low) if high != low else np.ones_like(f)
        mixed = (1.0 - blend) * f / factor + blend * f
        f = np.where(wl < original / high, f, np.where(wl > original / low, f / factor, mixed))
    elif sc:
        f = f / float(sc["factor"])
    return f.astype(np.float32)


def rotary_magnitude(rot: dict) -> float:
    """Factor on cosines and sines: 1 but for YaRN scaling, 0.1 ln(factor) + 1."""
    sc = rot.get("scaling")
    return 0.1 * math.log(float(sc["factor"])) + 1.0 if sc and "fast" in sc else 1.0
