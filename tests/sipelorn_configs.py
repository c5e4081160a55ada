"""Tiny Sipelorn configurations for tests: config.json dicts that differ in every size, constant and layer order."""


def attention(heads, kv_heads, dim, vdim, scale, conv=None, window=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if conv is not None:
        m["conv"] = conv
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, stretch=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
        if stretch is not None:
            factor, original, fast, slow = stretch
            m["rot"]["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# Every branch. Values narrower than keys, four query heads to a key head, a layer that reads the cache of one with a
# SHORTER window than its own, a reader that is itself followed by an owner, experts in three groups of which two are
# kept, a stretched rotation whose ramp covers part of the pairs, a layer without a feed-forward.
S_A = {"architecture": "Sipelorn", "vocab": 310, "width": 96, "norm": {"eps": 1e-5},
       "embedding": {"scale": 3.0, "bigram": {"buckets": 83, "mul_prev": 1009, "mul_cur": 31}}, "token_side": {"dim": 16},
       "layers": [
           layer("attention", attention(8, 2, 32, 16, 1.3, conv=4, window=21), moe(40, 6, 2, (3, 2), shared=56)),
           layer("attention", attention(4, 2, 32, 16, 0.9, conv=4, window=37, kv_from=0), dense(72)),
           layer("latent_attention", latent(3, 16, 16, 24, 40, 0.8, base=900.0, stretch=(6.0, 128, 16.0, 1.0)),
                 moe(24, 8, 3, (2, 1), shared=32)),
           layer("attention", attention(3, 3, 24, 24, 1.1, conv=2, window=16)),
           layer("latent_attention", latent(2, 24, 8, 16, 64, 1.5, base=5e4), dense(104)),
       ]}

# Odd sizes that defeat every vector path; no table of pairs, no token input, no convolution (a key left out) and one of a
# single tap, no window, no groups, no shared expert, a rotation of 6 numbers, a latent part that is not rotated at all.
S_B = {"architecture": "Sipelorn", "vocab": 259, "width": 70, "norm": {"eps": 1e-6},
       "layers": [
           layer("attention", attention(3, 3, 20, 12, 1.0, window=64), moe(17, 5, 5)),
           layer("latent_attention", latent(3, 12, 6, 20, 21, 1.1, base=300.0, stretch=(3.0, 64, 8.0, 2.0)), dense(33)),
           layer("attention", attention(5, 1, 12, 28, 1.4, conv=1), moe(9, 4, 1, (4, 2), shared=11)),
           layer("latent_attention", latent(2, 10, 0, 7, 9, 1.7), None),
           layer("attention", attention(2, 1, 12, 28, 0.7, conv=6, kv_from=2, window=5), moe(16, 2, 2, (2, 2))),
       ]}

# Heads of 64 and 128 as a served model has them, two layers that read one cache (one of them without a window, so its
# pages stay), a window of two pages and a half, wide experts.
S_C = {"architecture": "Sipelorn", "vocab": 512, "width": 128, "norm": {"eps": 1e-5},
       "embedding": {"scale": 1.0, "bigram": {"buckets": 1000, "mul_prev": 7, "mul_cur": 100003}}, "token_side": {"dim": 32},
       "layers": [
           layer("latent_attention", latent(4, 64, 32, 64, 128, 0.4, base=2e5, stretch=(4.0, 512, 32.0, 1.0)), dense(256)),
           layer("attention", attention(4, 2, 64, 64, 0.5, conv=4, window=160), moe(64, 4, 2, (2, 1), shared=64)),
           layer("attention", attention(4, 2, 64, 64, 0.5, conv=3, kv_from=1), moe(64, 4, 2, (2, 1), shared=64)),
           layer("attention", attention(2, 2, 64, 64, 0.4, conv=2, window=100, kv_from=1), moe(32, 8, 4, (4, 3))),
           layer("attention", attention(2, 1, 128, 128, 0.3, conv=4, window=65), moe(128, 3, 1, shared=192)),
       ]}

SIPELORN = {"sa": (S_A, 41), "sb": (S_B, 42), "sc": (S_C, 43)}

# models of one kind of layer alone
ONLY_LATENT = {"architecture": "Sipelorn", "vocab": 200, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
               "layers": [layer("latent_attention", latent(2, 32, 16, 32, 32, 1.0, base=1e4, stretch=(2.0, 32, 4.0, 1.0)), dense(64)),
                          layer("latent_attention", latent(4, 16, 8, 16, 48, 1.0), None)]}
ONLY_ATTENTION = {"architecture": "Sipelorn", "vocab": 200, "width": 64, "norm": {"eps": 1e-5},
                  "embedding": {"scale": 2.0, "bigram": {"buckets": 5, "mul_prev": 2, "mul_cur": 3}},
                  "layers": [layer("attention", attention(2, 1, 32, 32, 1.0, conv=4, window=7), moe(32, 2, 1)),
                             layer("attention", attention(2, 1, 32, 32, 1.0, conv=4, window=7, kv_from=0), dense(48))]}
ONE_KIND = {"latent": (ONLY_LATENT, 51), "attention": (ONLY_ATTENTION, 52)}
