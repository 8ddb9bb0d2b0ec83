"""Models of the Gebilorn design for the tests: small, with sizes that no two mechanisms share."""
from homura_b200 import synth

A, P, LA, R = synth.gebilorn_attention, synth.gebilorn_parallel, synth.gebilorn_latent, synth.gebilorn_rot
D, M = synth.gebilorn_dense, synth.gebilorn_moe

# name -> width of the decays' latents
RANKS = {"mixed": 12, "odd": 5, "ones": 1, "wide": 40, "far": 8, "large": 24, "windows": 6, "attention": 1, "latent": 1, "parallel": 16}


def model(name):
    """name -> config.json dict."""
    c = synth.gebilorn_config
    return {
        # every kind of mixer and feed-forward
        "mixed": lambda: c(96, 100, [
            (P((6, 3, 24, 40), 30, 3, (5, 16, 24), 8.0, (1.3, 0.6)), D(136)),
            (LA(5, 24, 12, 20, 56, 72), M(40, 7, 3, 56, 1.7)),
            (A(4, 2, 28, 36, 50, R(20, 1000.0, (3.0, 1.0, 4.0, 60.0)), 9, 0.6), M(24, 5, 2, 72, 0.8)),
            (P((2, 1, 40, 16), 70, 4, (3, 32, 8), 3.0), M(48, 6, 4, 32)),
            (LA(3, 16, 8, 48, 40, 40, R(8, 300.0)), None)], scale=0.2),
        # nothing is a multiple of four
        "odd": lambda: c(130, 77, [
            (P((5, 1, 11, 9), 13, 2, (3, 7, 5), 5.0, (0.7, 1.9)), D(33)),
            (LA(3, 9, 6, 11, 13, 29), M(35, 3, 2, 21, 1.3)),
            (A(9, 3, 13, 7, 21, R(6, 50.0), 3, 0.7), D(67))], 13, (5, 3), 1.7, 30.0, 1e-2),
        # one of everything
        "ones": lambda: c(17, 19, [
            (P((1, 1, 1, 1), 1, 1, (1, 1, 1), 1.0), M(1, 1, 1, 1)),
            (A(1, 1, 2, 1, 1, R(2, 10.0), 1), D(1)),
            (LA(1, 1, 2, 1, 1, 2), None)], 1, (1, 1), 1.0, 3.0, 1e-3),
        # more heads per key head than a tile of pairs, more experts than a mask word, wide feed-forwards
        "wide": lambda: c(320, 700, [
            (A(24, 2, 128, 80, 100, R(128, 10000.0, (4.0, 1.0, 4.0, 256.0)), 70), M(100, 40, 6, 200, 2.5)),
            (P((20, 4, 64, 40), 64, 5, (8, 64, 96), 16.0), D(700)),
            (LA(16, 64, 32, 64, 160, 128), M(64, 33, 30, 130))], 509),
        # sharp attention over long contexts: every key counts
        "far": lambda: c(64, 90, [
            (A(4, 2, 64, 32, 300, R(32, 10000.0, (4.0, 1.0, 4.0, 128.0)), 5, 0.4), D(48)),
            (LA(4, 32, 16, 32, 48, 64, scale=0.4), M(32, 4, 2, 24)),
            (P((4, 4, 32, 16), 128, 3, (4, 32, 32), 64.0, scale=0.4), None)]),
        # values above 128, heads above 256, linear states of several slices and lanes
        "large": lambda: c(72, 50, [
            (P((6, 2, 200, 160), 65, 3, (2, 96, 136)), M(24, 3, 1, 16)),
            (A(3, 1, 288, 272, 40, R(144), 64), D(40)),
            (P((2, 1, 48, 144), 64, 8, (1, 300, 20), 2.0), D(24)),
            (P((1, 1, 16, 16), 3, 2, (2, 20, 300)), None)]),
        # windows of every relation to the pages, kept tokens up to and beyond a page
        "windows": lambda: c(48, 60, [
            (A(2, 1, 16, 16, 64, R(8), 64, 1.0), None), (A(2, 2, 16, 24, 1, R(16), 2, 1.0), None), (A(4, 1, 24, 16, 63, R(2), 0, 0.8), D(32)),
            (A(2, 1, 16, 16, 65, R(8), 130, 1.0), None), (A(2, 1, 32, 16, 127, R(8), 1, 0.6), None), (P((2, 1, 16, 16), 64, 3, (2, 8, 8)), None)]),
        # one mixer by itself
        "attention": lambda: c(64, 80, [(A(4, 2, 32, 24, 40, R(16, 100.0, (2.0, 1.0, 4.0, 32.0)), 6), None)]),
        "latent": lambda: c(64, 80, [(LA(4, 24, 16, 32, 40, 48), None)]),
        "parallel": lambda: c(64, 80, [(P((4, 2, 24, 16), 20, 4, (4, 24, 16), 16.0, (0.8, 1.4)), None)]),
    }[name]()


NAMES = ["mixed", "odd", "ones", "wide", "far", "large", "windows", "attention", "latent", "parallel"]
