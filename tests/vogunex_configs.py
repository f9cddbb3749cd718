"""Small Vogunex configurations for tests: sizes that are not multiples of anything, single, grouped and odd head counts, value
widths of their own, rotations of part of a head, windows of one token and longer than a page, pooled blocks of one token, that
do and do not divide a page, and longer than the window, latents whose rotated part lies inside and behind the padded latent,
scans with one and several groups and norm parts, layers with another one's weights, with and without feed-forward."""
from ferrule_b200.models.layered_config import (CLAMPED_EXPERT, POOLED_WINDOW, PRE_NORM, DenseSpec, LatentMixer, LayeredConfig,
                                                LayerSpec, Mamba2Mixer, MoeSpec, WindowMixer)


def pooled(heads, kv_heads, dim, vdim, scale, window, pool, rot_dims=None, base=1000.0, softcap=9.0):
    return WindowMixer(heads, kv_heads, dim, vdim, scale, window, rot_base=base, rot_dims=dim // 2 * 2 if rot_dims is None else rot_dims,
                       softcap=softcap, pool=pool, **POOLED_WINDOW)


def latent(heads, dim, vdim, kv_rank, q_rank, rot_dim, window, scale=0.25, base=500.0):
    return LatentMixer(heads, dim, vdim, kv_rank, scale, q_rank, rot_dim, base, window)


def moe(experts, top, ff, limit, shared_ff, shared_limit):
    return MoeSpec(experts, top, ff, limit=limit, shared_ff=shared_ff, shared_limit=shared_limit, **CLAMPED_EXPERT)


def vogunex(vocab, width, eps, scale, *layers):
    return LayeredConfig(vocab, width, tuple(LayerSpec(*l) for l in layers), eps, name="vogunex", block=PRE_NORM, embed_scale=scale,
                         token_shift=True)


FF = DenseSpec(72, biases=True)
MOE = moe(5, 2, 24, 0.7, 40, 1.1)
CONFIGS = {
    "all": vogunex(
        97, 60, 1e-5, 1.5,
        (pooled(6, 3, 20, 12, 0.3, 9, 4, 8), FF),
        (latent(3, 12, 20, 26, 30, 6, 11), MOE),
        (pooled(6, 3, 20, 12, 0.3, 9, 4, 8), FF, 0),
        (Mamba2Mixer(4, 12, 10, 2, 3, 3), MOE),
        (pooled(4, 1, 16, 24, 0.4, 21, 7), None),
        (Mamba2Mixer(4, 12, 10, 2, 3, 3), MOE, 3),
        (latent(2, 16, 8, 40, 16, 16, 30), DenseSpec(33, biases=True))),
    "attention": vogunex(130, 64, 1e-6, 3.0, (pooled(20, 4, 24, 16, 0.2, 13, 5, 6), FF), (pooled(1, 1, 33, 10, 0.5, 1, 1), moe(4, 4, 16, 0.4, 8, 0.3)),
                         (pooled(2, 2, 64, 8, 0.2, 33, 40, 0, softcap=0.0), FF)),
    "latent": vogunex(80, 40, 1e-5, 1.0, (latent(4, 8, 8, 72, 24, 10, 5), FF), (latent(1, 24, 33, 15, 9, 2, 70), MOE)),
    "scan": vogunex(64, 48, 1e-6, 0.7, (Mamba2Mixer(3, 5, 3, 1, 1, 5), FF), (Mamba2Mixer(4, 16, 32, 2, 4, 2), moe(3, 1, 16, 2.0, 16, 2.0)),
                    (Mamba2Mixer(1, 72, 24, 1, 2), None)),
}
