"""Small Supisun configurations for tests: sizes that are not multiples of anything, grouped and single heads, unequal key
and value widths, partial rotation, chunks shorter and longer than a page, layers without feed-forward, one-tap
convolutions, layers without value mixing before, between and after mixing ones."""
from ferrule_b200.models.layered_config import (HEAD_DELTA, OUTPUT_NORM, AttentionMixer, DeltaMixer, DenseSpec, LayeredConfig,
                                                LayerSpec, MambaMixer)


def delta(heads, kv_heads, dim, vdim, taps):
    return DeltaMixer(heads, kv_heads, dim, vdim, taps, **HEAD_DELTA)


def supisun(vocab, width, taps, eps, *layers):
    return LayeredConfig(vocab_size=vocab, width=width, layers=tuple(LayerSpec(*l) for l in layers), norm_eps=eps, name="supisun",
                         max_position=700, block=OUTPUT_NORM, canon_taps=taps, learned_positions=True)


FF = DenseSpec(72)
CONFIGS = {
    "all": supisun(
        97, 52, 3, 1e-5,
        (AttentionMixer(6, 2, 20, 12, 0.3, 10, 5000.0, 12, False), FF),
        (AttentionMixer(4, 2, 12, 20, 0.5, 7, 100.0, 12, True), None),
        (MambaMixer(44, 5, 7, 4), DenseSpec(30)),
        (AttentionMixer(2, 2, 16, 20, 0.4, 24, 100.0, 8, True), FF),
        (delta(4, 2, 20, 12, 3), FF),
        (AttentionMixer(3, 1, 24, 8, 0.2, 16, 20.0, 2, False), FF),
        (AttentionMixer(6, 2, 10, 20, 0.4, 9, 1000.0, 6, True), DenseSpec(33))),
    "attention": supisun(
        130, 64, 4, 1e-6,
        (AttentionMixer(1, 1, 64, 64, 0.4, 19, 10000.0, 64, True), FF),
        (AttentionMixer(8, 1, 32, 64, 0.3, 33, 10000.0, 32, True), FF)),
    "mamba": supisun(80, 40, 1, 1e-5, (MambaMixer(70, 16, 3, 1), None), (MambaMixer(33, 20, 9, 6), DenseSpec(16))),
    "delta": supisun(80, 36, 5, 1e-5, (delta(6, 1, 8, 4, 1), FF), (delta(2, 2, 72, 33, 5), None)),
}
