"""Models of the Tunitar design for the tests: small, with sizes that no two mechanisms share."""
from homura_b200 import synth

L = synth.tunitar_layer


def model(name):
    """name -> config.json dict."""
    return {
        # layers without MLP, shared latents two layers apart, unequal head counts, a vocabulary below one slab
        "mixed": lambda: synth.tunitar_config(96, 100, [L(3, 24, 40, 72, None), L(2, 16, 16, 48, 56), L(5, 8, 24, 72, 88, kv_from=0, scale=0.9), L(1, 32, 8, 48, None, kv_from=1)], groups=3),
        # nothing is a multiple of four
        "odd": lambda: synth.tunitar_config(130, 77, [L(5, 11, 9, 65, 33, scale=0.7), L(3, 13, 7, 65, 35, kv_from=0)], groups=5, eps=1e-5),
        # one head, one group, one element where a size may be one
        "ones": lambda: synth.tunitar_config(16, 19, [L(1, 1, 1, 1, 1), L(1, 4, 3, 5, 7)], groups=1, eps=1e-3),
        # latents of five 64-element blocks, more heads than a tile of rows takes
        "wide": lambda: synth.tunitar_config(256, 700, [L(24, 32, 16, 320, 192, scale=0.5), L(40, 16, 32, 320, 128, kv_from=0, scale=0.6)], groups=16),
        # the widest latents the tensor-core kernel takes with several slices per tile
        "rank512": lambda: synth.tunitar_config(128, 260, [L(20, 64, 32, 512, 96, scale=0.3)], groups=2),
        # every element is its own group
        "unit_groups": lambda: synth.tunitar_config(48, 64, [L(2, 24, 24, 40, 48), L(4, 8, 16, 40, 24, kv_from=0)], groups=48, eps=0.02),
    }[name]()


NAMES = ["mixed", "odd", "ones", "wide", "rank512", "unit_groups"]
