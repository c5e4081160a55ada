"""Tiny Nisotar configurations for tests: config.json dicts that differ in every size, constant and layer order."""


def rotation(dims, base, stretch=None):
    rot = {"base": base, "dims": dims}
    if stretch is not None:
        factor, original, fast, slow = stretch
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return rot


def attention(heads, kv_heads, dim, vdim, scale, size=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = rotation(*rot)
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window=None, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot_dim:
        m["rot"] = rotation(rot_dim, base)
    return m


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
            "gate_rank": gate_rank}


def pair(left, right):
    return {"left": left, "right": right}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# Every branch. Chunks and windows off the pages' borders, two query heads to a key head on one side of a pair and four value
# heads to a query/key head on the other, values narrower than keys, a stretched rotation whose ramp covers part of the
# pairs, a whole head turned, a rotation alone without stretching, a layer without a feed-forward.
N_A = {"architecture": "Nisotar", "vocab": 301, "width": 104, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.5},
       "layers": [
           layer("parallel", pair(attention(4, 2, 32, 32, 0.7, 37, (32, 3000.0)), delta(4, 1, 24, 16, 3, 16, 8)), dense(88, 0.9)),
           layer("attention", attention(6, 3, 48, 32, 0.6, 21, (24, 900.0, (6.0, 128, 16.0, 1.0))), moe(40, 6, 3)),
           layer("latent_attention", latent(3, 16, 16, 24, 40, 1.2, 29), moe(24, 5, 1)),
           layer("parallel", pair(attention(2, 2, 16, 16, 1.1, 50, (8, 1e5)), delta(2, 2, 40, 32, 4, 24, 40))),
           layer("attention", attention(4, 1, 32, 32, 0.9, 64, (16, 5e4)), dense(56, 1.4)),
       ]}

# Odd sizes that defeat every vector path: inner vectors of 5 and 7 numbers, heads of 12, 20 and 21, one of them not turned,
# no window, no chunks, one tap, one expert, all experts a token, a latent part that is not turned at all.
N_B = {"architecture": "Nisotar", "vocab": 263, "width": 70, "norm": {"eps": 1e-6},
       "layers": [
           layer("attention", attention(3, 3, 20, 12, 1.0, None, (6, 300.0)), moe(17, 4, 4)),
           layer("parallel", pair(attention(5, 1, 12, 12, 1.3, 16, (2, 50.0)), delta(3, 3, 10, 7, 1, 5, 7)), moe(9, 3, 2)),
           layer("latent_attention", latent(3, 12, 6, 20, 21, 0.9, 17, 300.0), dense(33, 0.5)),
           layer("parallel", pair(attention(2, 1, 21, 21, 0.8), delta(4, 2, 33, 12, 6, 3, 9)), dense(19, 2.2)),
           layer("latent_attention", latent(2, 10, 0, 7, 9, 1.7), moe(16, 1, 1)),
           layer("attention", attention(2, 1, 28, 40, 0.9, 5)),
       ]}

# Heads of 64, 80 and 128 as a served model has them, chunks of two pages and a half and of exactly a page, a chunk of 128,
# a state of 128 rows, wide experts, a latent of 128 with a window of 65.
N_C = {"architecture": "Nisotar", "vocab": 520, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
       "layers": [
           layer("latent_attention", latent(4, 32, 32, 32, 128, 0.9, 65, 2e5), moe(64, 4, 2)),
           layer("parallel", pair(attention(4, 2, 64, 64, 0.3, 160, (64, 5e5)), delta(2, 1, 128, 64, 4, 32, 64)), moe(64, 8, 3)),
           layer("attention", attention(4, 2, 80, 80, 0.3, 100, (80, 1e4, (4.0, 512, 32.0, 1.0))), dense(256, 1.1)),
           layer("parallel", pair(attention(2, 1, 128, 128, 0.2, 64, (64, 7e4)), delta(4, 4, 64, 128, 2, 64, 16)), moe(128, 3, 1)),
           layer("attention", attention(6, 1, 64, 128, 0.25, 128, (32, 2e4)), dense(192, 0.8)),
       ]}

NISOTAR = {"na": (N_A, 61), "nb": (N_B, 62), "nc": (N_C, 63)}

# models of one kind of layer alone
ONLY_PAIRS = {"architecture": "Nisotar", "vocab": 210, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
              "layers": [layer("parallel", pair(attention(2, 1, 32, 32, 0.8, 24, (16, 500.0)), delta(2, 1, 16, 32, 4, 8, 8)), dense(40, 1.0)),
                         layer("parallel", pair(attention(2, 1, 32, 32, 0.8, 24, (16, 500.0)), delta(2, 1, 16, 32, 4, 8, 8)), moe(32, 2, 1))]}
ONLY_LATENT = {"architecture": "Nisotar", "vocab": 210, "width": 64, "norm": {"eps": 1e-5},
               "layers": [layer("latent_attention", latent(2, 32, 16, 32, 32, 1.0, 12), dense(64, 0.7)),
                          layer("latent_attention", latent(4, 16, 8, 16, 48, 1.0, 64), None)]}
ONLY_ATTENTION = {"architecture": "Nisotar", "vocab": 210, "width": 64, "norm": {"eps": 1e-5},
                  "layers": [layer("attention", attention(2, 1, 32, 32, 0.9, 7, (32, 1e4, (2.0, 32, 4.0, 1.0))), moe(32, 2, 1)),
                             layer("attention", attention(4, 4, 16, 16, 1.0, None), dense(48, 1.2))]}
ONE_KIND = {"pairs": (ONLY_PAIRS, 71), "latent": (ONLY_LATENT, 72), "attention": (ONLY_ATTENTION, 73)}


# Factors on the tensors of random weights: matrices of N(0, 0.02) would leave latent attention nearly uniform, its share of
# the stream small and the experts' weights equal.
LOUD = {".mix.dkv": 5.0, ".mix.uk": 5.0, ".mix.uv": 10.0, ".conv": 6.0, ".right.a1": 6.0, ".right.a2": 12.0, ".right.g1": 6.0,
        ".right.g2": 12.0, ".right.b": 8.0, ".router": 15.0, ".router.b": 8.0, ".gate": 4.0, ".up": 4.0, ".down": 4.0, ".gate.b": 4.0,
        ".up.b": 6.0, ".mix.o": 6.0}


def write_loud_folder(folder, cfg, seed, dtype):
    """A model folder with random weights in which every mechanism is loud enough for a fault to show."""
    import json
    import os
    from dynalm_b200.registry import find_architecture
    from dynalm_b200.weights.random_init import random_tensors
    from dynalm_b200.weights.safetensors import write_safetensors
    arch = find_architecture(cfg)
    tensors = random_tensors(arch.plan(arch.read_config(cfg)), seed)
    for name in tensors:
        factor = next((f for end, f in LOUD.items() if name.endswith(end)), 1.0)
        if ".mix.q" in name and name.replace(".q", ".dkv") in tensors:
            factor = 5.0                                # the queries of latent attention; others are normed anyway
        tensors[name] = (tensors[name].float() * factor).to(dtype)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
