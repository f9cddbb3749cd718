"""Small Vedadra configurations for tests: sizes that are not multiples of anything, single, grouped and odd head counts,
unequal map and value widths, windows shorter and longer than a page, windows of one token, kept tokens with and without,
norm parts that are and are not multiples of eight, loops of one layer, of all layers, of three passes, and no loop."""
from ferrule_b200.models.layered_config import (SANDWICH_NORM, TALKING_WINDOW, DenseSpec, LayeredConfig, LayerSpec, Loop,
                                                WindowMixer)


def talking(heads, kv_heads, dim, scale, window, keep_first=0):
    return WindowMixer(heads, kv_heads, dim, dim, scale, window, keep_first, **TALKING_WINDOW)


def differential(heads, kv_heads, dim, vdim, scale, window, keep_first, diff):
    return WindowMixer(heads, kv_heads, dim, vdim, scale, window, keep_first, maps=2, diff=diff)


def vedadra(vocab, width, groups, eps, loop, *layers):
    return LayeredConfig(vocab, width, tuple(LayerSpec(*l) for l in layers), eps, name="vedadra", block=SANDWICH_NORM,
                         norm_groups=groups, loop=Loop(*loop) if loop else None)


FF = DenseSpec(72, True)
CONFIGS = {
    "all": vedadra(
        97, 60, 3, 1e-5, (1, 4, 3),
        (talking(6, 3, 20, 0.3, 9), FF),
        (differential(4, 2, 12, 20, 0.5, 7, 3, 0.3), None),
        (talking(4, 4, 16, 0.4, 30, 5), DenseSpec(33, True)),
        (differential(3, 3, 10, 14, 0.4, 1, 1, 0.8), FF),
        (differential(2, 1, 24, 8, 0.2, 18, 0, 0.0), FF)),
    "talking": vedadra(130, 64, 1, 1e-6, (0, 2, 2), (talking(1, 1, 64, 0.2, 19), FF), (talking(8, 2, 40, 0.15, 33), None)),
    "differential": vedadra(80, 40, 5, 1e-5, None, (differential(6, 1, 16, 32, 0.4, 12, 20, 0.7), FF),
                            (differential(1, 1, 72, 33, 0.3, 25, 2, 0.45), None)),
    "once": vedadra(64, 48, 2, 1e-6, (1, 2, 1), (talking(2, 1, 8, 0.5, 4), FF), (talking(3, 1, 24, 0.4, 50), FF)),
}
