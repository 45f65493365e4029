"""Small Vogolix configurations for the tests (as config.json dictionaries).  Sizes differ from layer to layer and
include what a model may happen to make equal or 1: one head, key heads as many as query heads and fewer, values as
wide as keys and not, a rotation of fewer entries than a head has, one group of B and C or one per head, one norm
group or as many as heads, one tap, no feed-forward, chunks and windows shorter and longer than a page, layers that
share keys under the same chunk and under others, a factor of 1 on the logits."""

import copy
import random


def attention(heads, kv_heads, dim, vdim, size, rot_dims=None, base=10000.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
         "mask": {"size": size}, "rot": {"base": base, "dims": rot_dims if rot_dims is not None else dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, rank, size, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": size},
            "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}


def ssm(heads, vdim, state, groups=1, norm_groups=1, conv=4):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def model(layers, logit_scale=0.7, vocab=160, width=96, eps=1e-5):
    return {"architecture": "Vogolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for t, m, ff in layers]}


# every mechanism; two layers share the first one's keys, one of them under a longer chunk
MIX = model([
    ("attention", attention(4, 2, 32, 16, 50, rot_dims=8, scale=0.25), 112),
    ("mamba2", ssm(4, 16, 32, groups=2, norm_groups=2, conv=3), 80),
    ("latent_attention", latent(3, 16, 8, 24, 40, 37, scale=0.3), None),
    ("attention", attention(6, 2, 32, 16, 50, rot_dims=8, scale=0.2, kv_from=0), None),
    ("mamba2", ssm(6, 32, 16, groups=1, norm_groups=3, conv=4), None),
    ("attention", attention(2, 2, 32, 16, 83, rot_dims=8, scale=0.2, kv_from=0), 64),
    ("latent_attention", latent(2, 32, 16, 16, 48, 64, base=500.0), 96),
])

# sizes that are multiples of neither 8 nor 16; single heads; one tap; a group of B and C per head
ODD = model([
    ("mamba2", ssm(3, 7, 10, groups=3, norm_groups=1, conv=1), 52),
    ("attention", attention(3, 1, 22, 13, 19, rot_dims=6, base=50.0), None),
    ("latent_attention", latent(3, 10, 6, 9, 20, 11, base=100.0), 28),
    ("attention", attention(1, 1, 22, 13, 19, rot_dims=6, base=50.0, kv_from=1), 36),
    ("mamba2", ssm(1, 20, 7, groups=1, norm_groups=5, conv=2), None),
], vocab=130, width=100, logit_scale=1.0)

# one kind of mixer only
SPACES = model([("mamba2", ssm(2, 64, 48, groups=2, norm_groups=1, conv=4), None), ("mamba2", ssm(4, 32, 64, groups=1, norm_groups=4, conv=3), 64),
                ("mamba2", ssm(3, 80, 16, groups=3, norm_groups=3, conv=8), None)])
CHUNKS = model([("attention", attention(4, 4, 48, 32, 33, rot_dims=32), None),
                ("attention", attention(8, 4, 48, 32, 33, rot_dims=32, kv_from=0), 64),
                ("attention", attention(2, 1, 64, 64, 128, rot_dims=64, base=2e5), None),
                ("attention", attention(4, 4, 48, 32, 33, rot_dims=32, kv_from=0), None)], logit_scale=2.5)
WINDOWS = model([("latent_attention", latent(4, 16, 16, 16, 48, 21), None), ("latent_attention", latent(1, 32, 16, 64, 80, 129), 64),
                 ("latent_attention", latent(2, 16, 32, 32, 64, 1), None)])

ALL = {"mix": MIX, "odd": ODD, "spaces": SPACES, "chunks": CHUNKS, "windows": WINDOWS}


def one_layer(kind, mixer):
    return model([(kind, mixer, None)], vocab=48, width=64, logit_scale=1.3)


def clone(cfg):
    return copy.deepcopy(cfg)


def random_config(seed):
    """Layers of any kind in any order with sizes and constants drawn at random; attention layers may use an earlier
    one's keys, under its chunk or another."""
    r = random.Random(seed)
    layers, own = [], []
    for i in range(r.randint(3, 6)):
        kind = r.choice(["mamba2", "attention", "latent_attention"])
        if kind == "mamba2":
            groups = r.choice([1, 2, 3])
            heads = groups * r.choice([1, 2, 4])
            vdim = r.choice([8, 16, 20, 48, 64])
            mixer = ssm(heads, vdim, r.choice([8, 16, 24, 64, 80]), groups, r.choice([g for g in (1, 2, 4, heads) if heads * vdim % g == 0]),
                        r.choice([1, 2, 3, 4, 6]))
        elif kind == "attention":
            src = r.choice(own) if own and r.random() < 0.6 else None
            if src is None:
                g, dim, vdim = r.choice([1, 2, 3]), r.choice([16, 24, 32, 64]), r.choice([8, 16, 40, 64])
                dims, base, size = r.choice([d for d in (2, 8, 16, 24) if d <= dim]), r.choice([100.0, 1e4, 5e5]), r.choice([5, 16, 40, 100, 400])
                own.append(i)
            else:
                m = layers[src][1]
                g, dim, vdim, dims, base = m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"], m["rot"]["base"]
                size = r.choice([m["mask"]["size"], 7, 90])
            mixer = attention(g * r.choice([1, 2, 5]), g, dim, vdim, size, dims, base, r.choice([None, 0.2, 0.5]), src)
        else:
            mixer = latent(r.choice([1, 2, 5]), r.choice([8, 16, 24]), r.choice([2, 8, 16, 24]), r.choice([8, 16, 40]),
                           r.choice([16, 24, 48, 72]), r.choice([3, 16, 33, 120, 500]), r.choice([100.0, 1e4, 5e5]), r.choice([None, 0.2, 0.5]))
        layers.append((kind, mixer, r.choice([None, 16, 40, 96])))
    return model(layers, logit_scale=r.choice([0.25, 1.0, 3.0]), vocab=r.choice([100, 256]), width=r.choice([64, 96, 128]),
                 eps=r.choice([1e-6, 1e-5]))
