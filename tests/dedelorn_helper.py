"""Small Dedelorn models for the tests (own sizes, random weights)."""
import torch

from . import dedelorn_oracle as oracle
from .stack_helper import *  # noqa: F401,F403
from .stack_helper import DESIGNS


def delta(heads=6, kv=3, dim=20, vdim=28, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def latent(heads=3, dim=22, rot=10, vdim=36, rank=44, size=13, scale=0.21, base=300.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def dense(ff=76):
    return {"kind": "dense", "ff": ff}


def moe(ff=28, experts=7, top=3, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def config(layers, width=92, vocab=103, eps=2e-5):
    return {"architecture": "Dedelorn", "layers": [dict(m, mlp=f) for m, f in layers], "norm": {"eps": eps}, "vocab": vocab, "width": width}


#: unlike layers in one stack: sizes, windows, shared caches (two layers on one, a distant one), every feed-forward kind, one group
#: of heads and as many as heads
MIXED = config([(latent(), dense()),
                (delta(), moe()),
                (latent(heads=5, dim=40, rot=16, vdim=24, rank=48, size=70, base=5e4), None),
                (delta(heads=4, kv=4, dim=64, vdim=64, conv=4), dense(ff=40)),
                (latent(heads=4, dim=30, rot=10, vdim=50, size=40, scale=0.4, kv_from=0), moe(ff=20, experts=4, top=1, scale=0.6)),
                (delta(heads=3, kv=1, dim=16, vdim=8, conv=1), None),
                (latent(heads=2, dim=64, rot=16, vdim=64, rank=48, size=130, base=5e4, kv_from=2), dense(ff=64)),
                (latent(heads=2, dim=8, rot=10, vdim=12, size=1, kv_from=0), moe(ff=24, experts=9, top=4))])
#: sizes that are no multiples of 8 anywhere
ODD = config([(delta(heads=3, kv=3, dim=13, vdim=11, conv=5), dense(ff=37)),
              (latent(heads=3, dim=17, rot=6, vdim=13, rank=29, size=19), moe(ff=19, experts=5, top=2)),
              (delta(heads=4, kv=2, dim=7, vdim=10, conv=2), moe(ff=21, experts=3, top=3))], width=75, vocab=67, eps=3e-6)
#: heads wider than the 16-bit prompt kernels' tiles, a latent wider than the decode kernel's, no window at all
WIDE = config([(latent(heads=2, dim=130, rot=34, vdim=136, rank=600, size=None, scale=0.07), dense()),
               (delta(heads=2, kv=1, dim=150, vdim=96, conv=4), dense()),
               (latent(heads=3, dim=40, rot=24, vdim=40, rank=300, size=90, scale=0.11), None)], width=64, vocab=50)
#: everything a multiple of the tensor-core tiles: fused prompt paths, the chunked delta rule, the latent decode kernel
TILED = config([(delta(heads=4, kv=2, dim=128, vdim=128, conv=4), dense(ff=192)),
                (latent(heads=8, dim=96, rot=32, vdim=128, rank=256, size=150, scale=0.09), moe(ff=64, experts=8, top=2)),
                (delta(heads=6, kv=2, dim=96, vdim=64, conv=4), moe(ff=128, experts=4, top=2, scale=1.2)),
                (latent(heads=20, dim=32, rot=32, vdim=64, rank=256, size=300, scale=0.12, kv_from=1), dense(ff=256)),
                (latent(heads=4, dim=64, rot=64, vdim=64, rank=512, size=None, scale=0.08), dense(ff=128))], width=256, vocab=256)


def make_weights(cfg, seed, dtype, settled):
    """Random checkpoint tensors. Scales keep every branch audible in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, scale=None):
        return (torch.randn(shape, generator=g) * (shape[-1]**-0.5 if scale is None else scale)).to(dtype)

    def gain(n):
        return 1 + rnd(n, scale=0.2)

    w = {"embed": rnd(V, W, scale=1.0), "embed.norm": gain(W), "final.norm": gain(W), "head": rnd(V, W)}
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        q = p + "mix."
        w[p + "norm1"] = gain(W)
        if lc["type"] == "delta":
            kd, vd = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", kd), ("k", kd), ("v", vd)):
                w[q + n], w[q + n + ".conv"] = rnd(rows, W), rnd(rows, m["conv"], scale=0.6)
            w[q + "g"], w[q + "b"], w[q + "a"] = rnd(vd, W), rnd(m["heads"], W), rnd(m["heads"], W)
            w[q + "A_log"], w[q + "dt_bias"] = rnd(m["heads"], scale=1.0) - 1, rnd(m["heads"], scale=1.0) - 2
            w[q + "norm"], w[q + "o"] = gain(m["vdim"]), rnd(W, vd)
        else:
            w[q + "q"] = rnd(m["heads"] * (m["dim"] + m["rot_dim"]), W)
            if m.get("kv_from") is None:
                w[q + "dkv"], w[q + "dkv.norm"] = rnd(m["kv_rank"] + m["rot_dim"], W), gain(m["kv_rank"])
            w[q + "uk"], w[q + "uv"] = rnd(m["heads"] * m["dim"], m["kv_rank"]), rnd(m["heads"] * m["vdim"], m["kv_rank"])
            w[q + "o"] = rnd(W, m["heads"] * m["vdim"])
        f = lc["mlp"]
        if f is None:
            continue
        q = p + "mlp."
        if f["kind"] == "dense":
            w[q + "gate"], w[q + "up"], w[q + "down"] = rnd(f["ff"], W), rnd(f["ff"], W), rnd(W, f["ff"])
        else:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            w[q + "router"], w[q + "correction"] = rnd(n, W, scale=2 * W**-0.5), rnd(n, scale=0.3)
            if settled:       # corrections further apart than scores can be
                w[q + "correction"] = (1.5 * torch.randperm(n, generator=g)).to(dtype)
            for e in range(n):
                w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = rnd(ff, W), rnd(W, ff, scale=2 * ff**-0.5)
    return w


DESIGNS["Dedelorn"] = (make_weights, oracle)
