"""Models of the Dipisun design for the tests: small, with sizes that no two mechanisms share."""
from homura_b200 import synth

A, L = synth.dipisun_mixer, synth.dipisun_layer

# name -> rows of the distance tables
BUCKETS = {"mixed": 12, "odd": 7, "ones": 2, "wide": 24, "far": 32, "large_heads": 10}


def model(name):
    """name -> config.json dict."""
    return {
        # both kinds of attention, layers without a mixture, values blended from the second layer on, unequal experts
        "mixed": lambda: synth.dipisun_config(96, 100, [
            L(A(6, 3, 24, 40, 50, (0.7, 16)), 72, 5, 2, 3),
            L(A(4, 2, 16, 24, v_mix=True)),
            L(A(3, 1, 40, 48, 90, v_mix=True, scale=0.3), 40, 9, 0, 2, limit=0.5),
            L(A(8, 4, 32, 12, v_mix=True), 56, 3, 4, 5)]),
        # nothing is a multiple of four
        "odd": lambda: synth.dipisun_config(130, 77, [L(A(5, 1, 11, 9, 33, (0.5, 7), True, 0.7), 33, 3, 1, 2), L(A(9, 1, 13, 9, v_mix=True), 35, 7, 2, 1)], 1.3, 1e-2),
        # one of everything
        "ones": lambda: synth.dipisun_config(17, 19, [L(A(1, 1, 1, 1, 3, (1.0, 1)), 1, 1, 0, 1), L(A(1, 1, 3, 5), 5, 1, 1, 2)], 1.0, 1e-3),
        # more heads per key head than a tile of pairs, more experts than a mask word, most choices made
        "wide": lambda: synth.dipisun_config(320, 700, [L(A(24, 2, 128, 80, 200, (0.2, 40), True), 100, 40, 3, 6), L(A(20, 4, 64, 40, v_mix=True), 192, 33, 0, 30, limit=1.0)], 0.5),
        # sharp attention over long contexts: every key counts
        "far": lambda: synth.dipisun_config(64, 90, [L(A(4, 2, 64, 32, 100, (0.5, 64), True, 0.4), 48, 6, 2, 2), L(A(4, 4, 96, 16, v_mix=True, scale=0.3), 64, 4, 1, 1)], 0.7),
        # head sizes above 128 (wide value tiles) and above 256 (no tensor-core kernel), identity experts in the majority
        "large_heads": lambda: synth.dipisun_config(72, 50, [L(A(6, 2, 200, 160, 30), 24, 2, 6, 3), L(A(3, 1, 288, 272)), L(A(10, 1, 48, 144), 130, 4, 0, 4)], 0.4),
    }[name]()


NAMES = list(BUCKETS)
