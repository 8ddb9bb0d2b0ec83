"""Models of the Pulenex design for the tests: small, with sizes that no two mechanisms share."""
from homura_b200 import synth

RE, P, LA, R, D = synth.pulenex_retention, synth.pulenex_parallel, synth.pulenex_latent, synth.pulenex_rot, synth.pulenex_dense

# name -> widths of the latents of decays and of output gates
RANKS = {"mixed": (12, 20), "odd": (5, 3), "ones": (1, 1), "wide": (40, 130), "far": (8, 16), "large": (24, 9), "windows": (6, 4), "shared": (7, 7), "retention": (1, 1), "latent": (1, 1), "parallel": (16, 12)}


def model(name):
    """name -> config.json dict."""
    c = synth.pulenex_config
    return {
        # every kind of mixer, with and without a feed-forward
        "mixed": lambda: c(96, 100, [
            (P((6, 3, 24), 30, 3, (6, 2, 16, 24), 4, R(16, 1000.0)), D(136, 1.5)),
            (RE(5, 24, 40, R(16, 500.0)), None),
            (LA(5, 24, 12, 20, 72, 33), D(96, 2.0)),
            (RE(3, 16, 24), D(72, 0.5)),
            (LA(4, 16, 12, 28, 72, 50, 2, 300.0), None),
            (P((4, 1, 40), 70, 4, (3, 3, 32, 8), 2), None)], 0.7),
        # nothing is a multiple of four
        "odd": lambda: c(130, 77, [
            (P((5, 1, 11), 13, 2, (6, 3, 7, 5), 3, R(6, 50.0)), D(33, 0.7)),
            (LA(3, 9, 6, 11, 29, 17), D(67)),
            (RE(3, 13, 7, R(10, 100.0)), D(5, 1.0)),
            (P((9, 3, 13), 21, 5, (2, 1, 9, 3), 6, R(2)), None)], 1.9, 1e-2),
        # one of everything
        "ones": lambda: c(17, 19, [
            (P((1, 1, 2), 1, 1, (1, 1, 1, 1), 1), D(1, 0.25)),
            (RE(1, 2, 1, decay=[0.5]), D(1)),
            (LA(1, 1, 2, 1, 2, 1), None)], 3.0, 1e-3),
        # many heads, more heads per key head than an MMA has columns, wide feed-forwards
        "wide": lambda: c(320, 700, [
            (P((24, 2, 64), 100, 5, (16, 4, 64, 96), 5), D(700)),
            (LA(20, 64, 32, 64, 160, 64), D(130, 1.0)),
            (P((16, 16, 48), 64, 4, (8, 8, 32, 48), 4, R(32)), None),
            (RE(8, 64, 96, R(32)), D(200))], 0.5),
        # sharp attention over long contexts: every key counts
        "far": lambda: c(64, 90, [
            (P((4, 2, 64), 300, 3, (4, 2, 32, 32), 3, R(32), 0.5), D(48)),
            (LA(4, 32, 16, 32, 64, 400, scale=0.4), D(40, 2.0)),
            (RE(4, 32, 32, decay=[0.99, 0.999, 0.9995, 1.0]), None)]),
        # heads above 128, linear states of several slices and lanes
        "large": lambda: c(72, 50, [
            (P((3, 3, 200), 65, 3, (2, 1, 96, 136), 4, R(144)), D(40)),
            (RE(2, 96, 300, R(96)), D(24, 1.0)),
            (P((2, 1, 272), 64, 8, (1, 1, 300, 20), 2, R(16)), None),
            (LA(2, 200, 64, 136, 300, 70), None),
            (RE(1, 260, 24), None)]),
        # windows and chunks of every relation to the pages
        "windows": lambda: c(48, 60, [
            (LA(2, 16, 8, 16, 40, 64, scale=1.0), None), (LA(2, 16, 8, 16, 40, 1, 0, scale=1.0), None), (LA(3, 16, 8, 16, 40, 63, 0, scale=0.8), D(32)),
            (LA(2, 24, 8, 16, 24, 65, scale=1.0), None), (LA(2, 16, 8, 24, 24, 130, 3, scale=1.0), None), (P((2, 1, 16), 64, 3, (2, 1, 8, 8), 3, scale=1.0), None),
            (P((4, 2, 24), 1, 3, (1, 1, 8, 8), 3, R(8), 1.0), None), (P((2, 2, 16), 63, 2, (2, 2, 8, 8), 3, scale=0.8), None), (P((3, 1, 16), 130, 3, (2, 2, 8, 16), 3, R(8), 1.0), None)]),
        # latents that several layers read, with other heads, sizes and windows
        "shared": lambda: c(80, 70, [
            (LA(4, 16, 8, 24, 48, 30), None), (RE(2, 16, 16), D(48)), (LA(3, 24, 8, 16, 48, 90, 0), D(56)), (LA(5, 8, 12, 12, 36, 20), None),
            (LA(2, 32, 12, 8, 36, 5, 3), D(40)), (LA(6, 16, 8, 8, 48, 64, 0), None)]),
        # one mixer by itself
        "retention": lambda: c(64, 80, [(RE(4, 32, 24, R(16, 100.0)), None)]),
        "latent": lambda: c(64, 80, [(LA(4, 24, 16, 32, 48, 40), None)]),
        "parallel": lambda: c(64, 80, [(P((4, 2, 24), 40, 4, (4, 2, 24, 16), 3, R(16)), None)]),
    }[name]()


NAMES = ["mixed", "odd", "ones", "wide", "far", "large", "windows", "shared", "retention", "latent", "parallel"]
