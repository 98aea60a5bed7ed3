"""Frequency tables of rotary positions, formed once on the host in double precision (HybridLayer.rot_turns)."""
import math


def plain_frequencies(dims, base):
    """Radians per position of the dims/2 rotating pairs."""
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn(dims, base, factor, original, fast, slow):
    """YaRN: pairs that turn more than `fast` times over the `original` context keep their frequency, pairs that turn fewer than `slow` times
    are slowed down `factor` times, the ones between are blended linearly over the pair index.  -> (frequencies, amplitude of cosine and sine)."""
    def pair_of(turns):
        return dims * math.log(original / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    span = max(hi - lo, 0.001)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(1.0, max(0.0, (i - lo) / span))
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turns(frequencies):
    """Radians per position -> turns per position."""
    return [f / (2.0 * math.pi) for f in frequencies]
