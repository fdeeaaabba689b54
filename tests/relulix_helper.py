"""Small Relulix models for the tests (own sizes, random weights)."""
import torch

from . import relulix_oracle as oracle
from .stack_helper import *  # noqa: F401,F403
from .stack_helper import DESIGNS


def rotation(dims, base, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def retention(heads=3, dim=22, vdim=26, rot=12, base=700.0, decay=None, scaling=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": rotation(rot, base, scaling),
                                           "decay": decay or [1 - 2.0**-(1.5 + 1.3 * i) for i in range(heads)]}}


def attention(heads=6, kv=2, dim=20, vdim=28, rot=12, base=500.0, size=13, scale=0.3, softcap=4.0, scaling=(3.0, 40, 9.0, 0.7), kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rotation(rot, base, scaling), "scale": scale,
         "softcap": softcap}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def moe(ff=28, limit=1.3, experts=7, top=3):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=92, vocab=103, eps=2e-5, scale=1.7):
    return {"architecture": "Relulix", "embedding": {"scale": scale}, "layers": [dict(m, mlp=f) for m, f in layers], "norm": {"eps": eps},
            "vocab": vocab, "width": width}


#: unlike layers in one stack: sizes, windows down to one key, partly rotated heads, slowed rotations, layers on the keys and values
#: of one that is several layers back and with windows of their own, layers without feed-forward
MIXED = config([(retention(), moe()),
                (attention(), moe(ff=20, experts=4, top=1)),
                (attention(size=40, scale=0.2, softcap=9.0, kv_from=1), None),
                (retention(heads=2, dim=40, vdim=18, rot=40, base=5e4, decay=[0.9, 1.0], scaling=(2.0, 64, 8.0, 1.0)), None),
                (attention(heads=4, kv=4, dim=70, vdim=24, rot=70, base=5e4, size=130, scale=0.15, scaling=(8.0, 300, 32.0, 1.0)), moe()),
                (attention(size=1, kv_from=1), moe(ff=24, experts=9, top=4, limit=0.4)),
                (retention(heads=5, dim=16, vdim=48, rot=2), moe(experts=3, top=3)),
                (attention(heads=8, kv=4, dim=70, vdim=24, rot=70, base=5e4, size=33, scale=0.1, scaling=(8.0, 300, 32.0, 1.0), kv_from=4), None)])
#: sizes that are no multiples of 8 anywhere
ODD = config([(attention(heads=9, kv=3, dim=15, vdim=21, rot=14, size=33, scaling=None), moe(ff=19, experts=5, top=2)),
              (retention(heads=3, dim=7, vdim=9, rot=6), moe(ff=21, experts=3, top=3)),
              (attention(heads=3, kv=3, dim=17, vdim=21, rot=10, size=19), None),
              (attention(heads=9, kv=3, dim=15, vdim=21, rot=14, size=8, scaling=None, kv_from=0), moe(ff=23, experts=6, top=1))],
             width=75, vocab=67, eps=3e-6)
#: heads wider than the 16-bit kernels' tiles, many query heads on one key head, more key channels than the chunked recurrence takes
WIDE = config([(attention(heads=12, kv=1, dim=130, vdim=136, rot=34, size=90, scale=0.07), moe()),
               (retention(heads=1, dim=272, vdim=150, rot=272), None),
               (attention(heads=10, kv=1, dim=130, vdim=136, rot=34, size=20, scale=0.07, kv_from=0), moe(ff=40)),
               (attention(heads=2, kv=1, dim=60, vdim=136, rot=60, size=50), moe(ff=40))], width=64, vocab=50)
#: everything a multiple of the tensor-core tiles: fused prompt paths, packed decode, the chunked recurrences
TILED = config([(retention(heads=4, dim=64, vdim=128, rot=64), moe(ff=64, experts=8, top=2)),
                (attention(heads=8, kv=2, dim=128, vdim=96, rot=128, base=1e5, size=150, scale=0.12, softcap=12.0, scaling=(4.0, 256, 16.0, 1.0)), None),
                (attention(heads=6, kv=2, dim=64, vdim=96, rot=32, size=300), moe(ff=128, experts=4, top=2)),
                (attention(heads=12, kv=2, dim=64, vdim=96, rot=32, size=100, kv_from=2), moe(ff=96, experts=4, limit=0.7)),
                (retention(heads=2, dim=128, vdim=48, rot=64, base=1e5), moe(ff=64, experts=8, top=1)),
                (attention(heads=4, kv=2, dim=64, vdim=64, rot=48, size=64), None),
                (retention(heads=2, dim=32, vdim=256, rot=32, decay=[0.999, 0.3]), None)], width=256, vocab=256)


def make_weights(cfg, seed, dtype, settled):
    """Random checkpoint tensors. Scales keep every branch audible in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, scale=None):
        return (torch.randn(shape, generator=g) * (shape[-1]**-0.5 if scale is None else scale)).to(dtype)

    def gain():
        return (1 + torch.randn((), generator=g) * 0.2).to(dtype)

    w = {"embed": rnd(V, W, scale=1.0), "final.norm": gain(), "head": rnd(V, W)}
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        q = p + "mix."
        w[p + "norm1"] = gain()
        n_o = m["heads"] * m["vdim"]
        w[q + "o"] = rnd(W, n_o, scale=2 * n_o**-0.5)
        if lc["type"] == "retention":
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["heads"] * m["dim"]), ("v", n_o), ("g", n_o)):
                w[q + n] = rnd(rows, W)
            if settled:       # (a token's own key answers its query: no head's output is so small that its norm magnifies rounding)
                w[q + "k"] = (0.8 * w[q + "q"].float() + 0.6 * w[q + "k"].float()).to(dtype)
        else:
            own = [("q", m["heads"] * m["dim"])]
            if m.get("kv_from") is None:
                own += [("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])]
            for n, rows in own:
                w[q + n], w[q + n + ".b"] = rnd(rows, W), rnd(rows, scale=0.3)
        f = lc["mlp"]
        if f is None:
            continue
        q = p + "mlp."
        n, ff = f["router"]["experts"], f["expert"]["ff"]
        w[q + "router"], w[q + "router.b"] = rnd(n, W, scale=2 * W**-0.5), rnd(n, scale=0.5)
        like = {"gate": rnd(ff, W), "up": rnd(ff, W), "down": rnd(W, ff, scale=2 * ff**-0.5)}
        for e in range(n):
            for x, t in like.items():
                own = rnd(*t.shape, scale=(2 if x == "down" else 1) * t.shape[1]**-0.5)
                # (settled: experts so alike that a choice which rounding decides makes no difference to speak of)
                w[f"{q}e{e}.{x}"] = t + own * 0.05 if settled else own
    return w


DESIGNS["Relulix"] = (make_weights, oracle)
