"""Small Lakatar configurations for the tests (as config.json dictionaries).  Sizes differ from layer to layer and
include what a model may happen to make equal or 1: one head, values as wide as keys and not, a rotation of fewer
entries than a head has, one group of experts, every group kept, one expert chosen or all of them, no shared
expert, no feed-forward, a latent that two layers share and one of its own between them, no YaRN scaling, a
stretch of 1."""

import copy
import random


def wkv(heads, dim, rank):
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def retention(heads, dim, vdim, rot_dims=None, base=10000.0, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims if rot_dims is not None else dim},
            "decay": decay if decay is not None else [1.0 - 2.0 ** -(2 + 1.5 * h) for h in range(heads)]}


def latent(heads, dim, rot_dim, vdim, rank, q_rank, base=10000.0, scale=None, scaling=(4.0, 64, 8.0, 1.0), kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
         "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(experts, top, ff, groups=(1, 1), scale=1.0, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups[0], "keep": groups[1]}}}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def model(layers, alpha=1.8, vocab=160, width=96, eps=1e-5):
    return {"architecture": "Lakatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}


def _mix(calm):
    def routed(experts, top, ff, groups, scale, shared):
        return moe(experts, experts if calm else top, ff, (groups[0], groups[0]) if calm else groups, scale, shared)
    return model([
        ("latent_attention", latent(3, 16, 8, 24, 40, 48, scale=0.25), routed(6, 2, 40, (3, 2), 1.5, 24)),
        ("wkv", wkv(3, 16, 8), routed(4, 1, 32, (2, 1), 2.0, 72)),
        ("latent_attention", latent(2, 24, 16, 16, 32, 24, base=500.0, scaling=None), None),
        ("retention", retention(2, 32, 48, rot_dims=16), routed(8, 3, 24, (4, 2), 0.5, None)),
        ("latent_attention", latent(5, 8, 8, 40, 40, 32, scale=0.3, kv_from=0), routed(4, 2, 48, (1, 1), 1.0, 16)),
        ("wkv", wkv(2, 48, 16), None),
    ])


# every mechanism
MIX = _mix(False)
# the same with routers that choose every expert (no close calls): for 16-bit engines
CALM = _mix(True)


# sizes that are multiples of neither 8 nor 16; single heads; one expert
def _odd(calm):
    return model([
        ("wkv", wkv(3, 7, 5), moe(6, 6 if calm else 2, 28, (3, 3 if calm else 1), 0.7, 20)),
        ("latent_attention", latent(3, 10, 6, 12, 20, 18, base=100.0, scaling=(2.5, 30, 4.0, 0.5)), None),
        ("retention", retention(1, 10, 13, rot_dims=6), moe(1, 1, 12, (1, 1), 3.0, None)),
        ("retention", retention(3, 22, 5, rot_dims=22, base=50.0), moe(5, 5 if calm else 3, 20, (5, 5 if calm else 4), 1.0, 9)),
        ("latent_attention", latent(1, 5, 6, 9, 20, 11, base=100.0, scaling=(2.5, 30, 4.0, 0.5), kv_from=1), None),
    ], vocab=130, width=100, alpha=1.0)


ODD, ODD_CALM = _odd(False), _odd(True)

# one kind of mixer only
WKVS = model([("wkv", wkv(2, 32, 24), None), ("wkv", wkv(1, 64, 8), moe(2, 2, 32, (1, 1), 1.0, 48)), ("wkv", wkv(4, 16, 16), None)], alpha=2.2)
RETENTIONS = model([("retention", retention(4, 16, 16), None),
                    ("retention", retention(2, 64, 96, rot_dims=32, decay=[0.5, 0.999]), moe(2, 2, 32, (2, 2), 1.0, None))], alpha=1.5)
LATENTS = model([("latent_attention", latent(4, 16, 16, 16, 48, 64, scale=0.35), None),
                 ("latent_attention", latent(1, 32, 16, 64, 48, 32, kv_from=0), moe(3, 3, 64, (3, 3), 0.8, 32)),
                 ("latent_attention", latent(2, 16, 32, 32, 64, 48, scaling=(1.0, 100, 32.0, 1.0)), None),
                 ("latent_attention", latent(2, 16, 16, 8, 48, 40, kv_from=0), None)])

ALL = {"mix": MIX, "calm": CALM, "odd": ODD, "odd_calm": ODD_CALM, "wkvs": WKVS, "retentions": RETENTIONS, "latents": LATENTS}


def one_latent_layer(heads=2, dim=16, rot_dim=8, vdim=16, rank=32, q_rank=32):
    return model([("latent_attention", latent(heads, dim, rot_dim, vdim, rank, q_rank, base=200000.0), None)], vocab=48, width=64,
                 alpha=0.7)


def one_layer(kind, mixer):
    return model([(kind, mixer, None)], vocab=48, width=64, alpha=0.7)


def clone(cfg):
    return copy.deepcopy(cfg)


def random_config(seed, calm=False):
    """Layers of any kind in any order with sizes and constants drawn at random; latent layers may share an earlier
    one's latent."""
    r = random.Random(seed)
    layers, own = [], []
    for i in range(r.randint(3, 6)):
        kind = r.choice(["wkv", "retention", "latent_attention"])
        if kind == "wkv":
            mixer = wkv(r.choice([1, 2, 5]), r.choice([8, 16, 20, 40, 64]), r.choice([4, 8, 24]))
        elif kind == "retention":
            dim = r.choice([8, 16, 24, 64])
            heads = r.choice([1, 2, 3])
            mixer = retention(heads, dim, r.choice([8, 16, 40, 64]), rot_dims=r.choice([d for d in (2, 8, 16, 64) if d <= dim]),
                              base=r.choice([100.0, 1e4, 5e5]), decay=[r.choice([0.3, 0.9, 0.99, 0.9995]) for _ in range(heads)])
        else:
            src = r.choice(own) if own and r.random() < 0.5 else None
            if src is None:
                rank, rot_dim, base = r.choice([16, 24, 48, 72]), r.choice([2, 8, 16, 24]), r.choice([100.0, 1e4, 5e5])
                scaling = r.choice([None, (4.0, 64, 8.0, 1.0), (16.0, 512, 32.0, 2.0)])
                own.append(i)
            else:
                m = layers[src][1]
                rank, rot_dim, base = m["kv_rank"], m["rot_dim"], m["rot"]["base"]
                scaling = tuple(m["rot"]["scaling"].values()) if "scaling" in m["rot"] else None
            mixer = latent(r.choice([1, 2, 5]), r.choice([8, 16, 24]), rot_dim, r.choice([8, 16, 40]), rank, r.choice([16, 24, 40]),
                           base=base, scale=r.choice([None, 0.2, 0.5]), scaling=scaling, kv_from=src)
        mlp = None
        if r.random() < 0.75:
            count = r.choice([1, 2, 3])
            experts = count * r.choice([1, 2, 3])
            keep = count if calm else r.randint(1, count)
            mlp = moe(experts, experts if calm else r.randint(1, keep * (experts // count)), r.choice([16, 40]), (count, keep),
                      r.choice([0.5, 1.0, 2.5]), r.choice([None, 16, 48]))
        layers.append((kind, mixer, mlp))
    return model(layers, alpha=r.choice([1.0, 1.7, 3.0]), vocab=r.choice([100, 256]), width=r.choice([64, 96, 128]),
                 eps=r.choice([1e-6, 1e-5]))
