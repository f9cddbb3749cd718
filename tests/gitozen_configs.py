"""Small Gitozen configurations for tests: sizes that are not multiples of anything, grouped and single heads, layers
without feed-forward, one-tap convolutions, one expert group and one expert per group."""
from ferrule_b200.models.layered_config import DeltaMixer, LatentMixer, LayeredConfig, LayerSpec, MoeSpec

MOE = MoeSpec(experts=6, top=2, ff=24, groups=3, keep=2)
CONFIGS = {
    "both": LayeredConfig(vocab_size=97, width=52, layers=(
        LayerSpec(DeltaMixer(4, 2, 20, 12, 3, 6, 10), MOE),
        LayerSpec(LatentMixer(3, 20, 12, 36, 0.4), MOE),
        LayerSpec(DeltaMixer(3, 3, 12, 40, 4, 8, 8), None),
        LayerSpec(LatentMixer(5, 8, 24, 72, 0.7), MoeSpec(4, 1, 40, 4, 1))), norm_eps=1e-5, logit_softcap=6.0),
    "latent": LayeredConfig(vocab_size=130, width=64, layers=(
        LayerSpec(LatentMixer(1, 16, 16, 64, 1.2), None),
        LayerSpec(LatentMixer(4, 32, 20, 130, 0.3), MoeSpec(8, 3, 32)))),
    "delta": LayeredConfig(vocab_size=80, width=40, layers=(
        LayerSpec(DeltaMixer(6, 1, 8, 4, 1, 4, 4), MoeSpec(5, 2, 8)),
        LayerSpec(DeltaMixer(2, 2, 72, 33, 5, 9, 7), None)), logit_softcap=3.0),
}
