"""Small Gozolix configurations for the tests. Every size differs between them and from layer to
layer, and some take the values that make branches coincide elsewhere: one head, as many
key/value heads as heads and fewer (in both mixers), values wider and narrower than keys,
convolutions of one tap (no running inputs at all) and of many, keys of four numbers and wider than
a warp's lanes hold eight each, query temperatures whose steps fall inside a cache block, at its
border and never, and none, caps that bind and none, layers that read another's keys and values
(one after the other, and with layers between), experts in one group, in several and in groups of
one, with and without a shared expert, one choice and as many as open experts, layers without a
feed-forward, a table of pairs that is small, large and absent, the kinds of layers in any order,
and sizes that no vector access divides."""


def delta(heads, kv_heads, dim, vdim, taps, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim,
                                       "vdim": vdim, "conv": taps}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, cap, temp, mlp, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap is not None:
        mixer["softcap"] = cap
    if temp is not None:
        mixer["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, shared=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def bigram(buckets, mul_prev, mul_cur):
    return {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}


MIXED = {"architecture": "Gozolix", "vocab": 211, "width": 96, "norm": {"eps": 1e-5},
         "embedding": {"scale": 2.5, "bigram": bigram(101, 13, 5)}, "initializer_range": 0.1,
         "layers": [attention(4, 2, 32, 24, 0.25, 4.0, (0.4, 37), dense(80)),
                    delta(6, 3, 24, 16, 4, moe(8, 3, 48, (4, 2), 56, 2.0)),
                    attention(4, 2, 32, 24, 0.4, None, None, moe(6, 2, 40, (3, 1), None, 0.7), 0),
                    delta(4, 4, 16, 40, 3, None),
                    attention(6, 1, 48, 16, 0.2, 10.0, (0.2, 64), None),
                    attention(6, 1, 48, 16, 0.5, 2.5, (0.3, 5), dense(130), 4),
                    attention(4, 2, 32, 24, 0.3, 7.0, (0.6, 100), dense(64), 0)]}
ODD = {"architecture": "Gozolix", "vocab": 131, "width": 100, "norm": {"eps": 3e-6},
       "embedding": {"scale": 1.0, "bigram": bigram(7, 3, 2)}, "initializer_range": 0.12,
       "layers": [delta(5, 1, 20, 12, 1, moe(9, 1, 22, (9, 2), 30)),
                  delta(3, 3, 7, 10, 6, dense(30)),
                  attention(5, 5, 12, 20, 0.7, 1.5, (0.25, 1), moe(5, 5, 50)),
                  attention(1, 1, 36, 28, 0.3, 6.0, None, moe(6, 4, 34, (2, 2), 18, 3.0)),
                  delta(1, 1, 4, 50, 2, None),
                  attention(5, 5, 12, 20, 0.2, None, (1.5, 1000), None, 2)]}
WIDE = {"architecture": "Gozolix", "vocab": 97, "width": 128, "norm": {"eps": 1e-6},
        "embedding": {"scale": 4.0}, "initializer_range": 0.07,
        "layers": [delta(4, 2, 128, 128, 4, dense(256)),
                   delta(2, 1, 256, 64, 5, moe(16, 4, 128, (8, 3), 128, 2.5)),
                   attention(4, 1, 128, 128, 0.088, 30.0, (0.1, 128), moe(4, 4, 32, (2, 2))),
                   delta(8, 4, 64, 48, 2, None),
                   attention(2, 2, 64, 320, 0.125, 5.0, (0.6, 200), dense(72))]}
CONFIGS = {"mixed": (MIXED, 61), "odd": (ODD, 62), "wide": (WIDE, 63)}
