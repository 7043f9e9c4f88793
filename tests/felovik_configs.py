"""Small Felovik configurations for the tests. Every size differs between them and from layer to
layer, and some take the values that make branches coincide elsewhere: one head, as many
key/value heads as heads and fewer, values wider and narrower than keys, as many groups of B and
C as heads and one, one norm part and many, a convolution of one tap (no running inputs at all)
and of many, a state of one number and one wider than a warp's lanes hold four each, query
temperatures whose steps fall inside a block, at its border and never, and none, experts in one
group, in several and in groups of one, as many open groups as there are, one choice and as
many as open experts, a limit that binds and one that never does, layers without a
feed-forward, and sizes that no vector access divides."""


def left(heads, kv_heads, dim, vdim, scale, temp):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        out["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return out


def right(heads, vdim, state, groups, taps, parts):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps,
            "norm_groups": parts}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff}}


def layer(a, b, mlp):
    return {"type": "parallel", "mixer": {"left": left(*a), "right": right(*b)}, "mlp": mlp}


MIXED = {"architecture": "Felovik", "vocab": 211, "width": 96, "max_positions": 640,
         "norm": {"eps": 1e-5}, "embedding": {"scale": 2.5}, "postln_alpha": 2.0,
         "initializer_range": 0.1,
         "layers": [layer((4, 2, 32, 24, 0.25, (0.4, 37)), (4, 16, 24, 2, 4, 2), dense(80, 0.6)),
                    layer((6, 3, 16, 40, 0.5, (0.2, 64)), (3, 24, 16, 1, 3, 1),
                          moe(8, 3, 48, (4, 2))),
                    layer((2, 1, 48, 16, 0.3, None), (6, 8, 40, 3, 2, 6), None),
                    layer((3, 3, 24, 32, 1.0, (0.3, 5)), (2, 40, 8, 2, 5, 4),
                          moe(5, 2, 40))]}
ODD = {"architecture": "Felovik", "vocab": 131, "width": 100, "max_positions": 700,
       "norm": {"eps": 3e-6}, "embedding": {"scale": 1.0}, "postln_alpha": 0.7,
       "initializer_range": 0.12,
       "layers": [layer((6, 2, 20, 12, 0.4, (0.5, 3)), (5, 12, 7, 5, 3, 5),
                        moe(9, 1, 22, (9, 2))),
                  layer((5, 1, 12, 20, 0.7, (0.25, 100)), (3, 10, 1, 1, 1, 3), dense(30, 1.1)),
                  layer((1, 1, 36, 28, 0.2, None), (1, 50, 30, 1, 7, 10), None),
                  layer((4, 4, 10, 6, 0.9, (1.5, 1000)), (6, 6, 36, 2, 2, 4),
                        moe(6, 4, 50, (3, 2)))]}
WIDE = {"architecture": "Felovik", "vocab": 97, "width": 128, "max_positions": 1024,
        "norm": {"eps": 1e-6}, "embedding": {"scale": 4.0}, "postln_alpha": 3.5,
        "initializer_range": 0.07,
        "layers": [layer((4, 1, 128, 128, 0.088, (0.1, 128)), (4, 64, 128, 1, 4, 1),
                         dense(256, 7.0)),
                   layer((2, 2, 64, 320, 0.125, (0.6, 200)), (2, 64, 160, 2, 4, 2),
                         moe(16, 4, 128, (8, 3))),
                   layer((6, 2, 64, 48, 0.15, None), (8, 32, 64, 4, 4, 8),
                         moe(4, 4, 32, (2, 2)))]}
CONFIGS = {"mixed": (MIXED, 51), "odd": (ODD, 52), "wide": (WIDE, 53)}
