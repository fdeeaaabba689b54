"""Small Lotelix models for the tests (own sizes, random weights)."""
import torch

from . import lotelix_oracle as oracle
from .stack_helper import *  # noqa: F401,F403
from .stack_helper import DESIGNS


def gru(width=70):
    return {"type": "mingru", "mixer": {"width": width}}


def attention(heads=6, kv=2, dim=20, vdim=28, rot=12, base=500.0, size=13, scale=0.3, v_mix=False, scaling=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": r, "scale": scale,
                                           "v_mix": v_mix}}


def parallel(heads=3, kv=3, dim=22, vdim=36, rot=22, base=900.0, scale=0.2, lin=2, ldim=10, lvdim=18, tau=3.0, rank=5):
    """(``rank`` is no key of a config: the checkpoint's tensors have it.)"""
    return {"type": "parallel", "rank": rank,
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "scale": scale},
                      "right": {"heads": lin, "dim": ldim, "vdim": lvdim, "tau": tau}}}


def moe(ff=28, experts=7, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=92, vocab=103, eps=2e-5, groups=4, scale=1.7):
    return {"architecture": "Lotelix", "embedding": {"scale": scale}, "layers": [dict(m, mlp=f) for m, f in layers],
            "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


#: unlike layers in one stack: sizes, windows down to one key, partly rotated heads, slowed rotations, values mixed over layers of
#: different page sizes and around a layer that does not mix, layers without feed-forward
MIXED = config([(gru(), moe()),
                (attention(), moe(ff=20, experts=4, top=1)),
                (parallel(), None),
                (attention(heads=4, dim=24, vdim=24, rot=24, size=40, v_mix=True, scaling=(8.0, 1.0, 4.0, 64)), moe()),
                (gru(width=96), None),
                (attention(heads=2, dim=40, vdim=24, rot=8, size=1, v_mix=True), moe(ff=24, experts=9, top=4)),
                (attention(heads=8, dim=70, vdim=24, rot=70, base=5e4, size=130, scale=0.15, v_mix=True, scaling=(3.0, 0.5, 6.0, 300)), None),
                (parallel(heads=4, kv=1, dim=30, vdim=16, rot=6, base=5e4, lin=3, ldim=24, lvdim=40, tau=11.0, rank=12), moe(experts=3, top=3))])
#: sizes that are no multiples of 8 anywhere
ODD = config([(parallel(heads=3, kv=1, dim=13, vdim=11, rot=6, lin=3, ldim=7, lvdim=9, tau=1.5, rank=3), moe(ff=19, experts=5, top=2)),
              (gru(width=37), moe(ff=21, experts=3, top=3)),
              (attention(heads=3, kv=3, dim=17, vdim=21, rot=10, size=19, v_mix=True), None),
              (attention(heads=9, kv=3, dim=15, vdim=21, rot=14, size=33, v_mix=True), moe(ff=23, experts=6, top=1))],
             width=75, vocab=67, eps=3e-6, groups=5)
#: heads wider than the 16-bit kernels' tiles, many query heads on one key head, more key channels than the chunked recurrence takes
WIDE = config([(attention(heads=12, kv=1, dim=130, vdim=136, rot=34, size=90, scale=0.07, v_mix=True), moe()),
               (parallel(heads=10, kv=1, dim=140, vdim=40, rot=140, scale=0.05, lin=1, ldim=272, lvdim=150, tau=5.0, rank=20), None),
               (attention(heads=2, kv=1, dim=60, vdim=136, rot=60, size=20, v_mix=True), moe(ff=40))], width=64, vocab=50, groups=1)
#: everything a multiple of the tensor-core tiles: fused prompt paths, packed decode, the chunked recurrences
TILED = config([(gru(width=320), moe(ff=64, experts=8, top=2)),
                (parallel(heads=8, kv=2, dim=128, vdim=128, rot=64, scale=0.09, lin=4, ldim=64, lvdim=128, tau=16.0, rank=16), moe(ff=96, experts=4)),
                (attention(heads=8, kv=2, dim=128, vdim=96, rot=128, base=1e5, size=150, scale=0.12, v_mix=True, scaling=(4.0, 1.0, 4.0, 256)), None),
                (attention(heads=6, kv=2, dim=64, vdim=96, rot=32, size=300, v_mix=True), moe(ff=128, experts=4, top=2)),
                (parallel(heads=4, kv=4, dim=64, vdim=64, rot=64, lin=2, ldim=128, lvdim=48, tau=2.0, rank=24), moe(ff=64, experts=8, top=1)),
                (attention(heads=4, kv=2, dim=64, vdim=64, rot=48, size=64), None)], width=256, vocab=256, groups=2)


def make_weights(cfg, seed, dtype, settled):
    """Random checkpoint tensors. Scales keep every branch audible in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, scale=None):
        return (torch.randn(shape, generator=g) * (shape[-1]**-0.5 if scale is None else scale)).to(dtype)

    def gain(n):
        return 1 + rnd(n, scale=0.2)

    w = {"embed": rnd(V, W, scale=1.0), "final.norm": gain(W), "head": rnd(V, W)}
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        q = p + "mix."
        w[p + "norm1"] = gain(W)
        if lc["type"] == "mingru":
            C = m["width"]
            w[q + "z"], w[q + "z.b"], w[q + "x"], w[q + "x.b"] = rnd(C, W), rnd(C, scale=0.5) - 1, rnd(C, W), rnd(C, scale=0.5)
            w[q + "g"], w[q + "o"] = rnd(C, W), rnd(W, C, scale=2 * C**-0.5)
        elif lc["type"] == "attention":
            w[q + "q"], w[q + "k"] = rnd(m["heads"] * m["dim"], W), rnd(m["kv_heads"] * m["dim"], W)
            w[q + "v"], w[q + "g"] = rnd(m["kv_heads"] * m["vdim"], W), rnd(m["heads"] * m["vdim"], W)
            w[q + "sink"], w[q + "o"] = rnd(m["heads"], scale=1.0) + 1, rnd(W, m["heads"] * m["vdim"], scale=2 * (m["heads"] * m["vdim"])**-0.5)
            if m["v_mix"]:
                w[q + "vmix"] = rnd(1, scale=0.2)[0] + 0.5
        else:
            a, r = m["left"], m["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                w[q + "left." + n], w[q + "left." + n + ".b"] = rnd(rows, W), rnd(rows, scale=0.3)
            w[q + "left.q.norm"], w[q + "left.k.norm"] = gain(a["heads"] * a["dim"]), gain(a["kv_heads"] * a["dim"])
            w[q + "left.pb"] = rnd(a["heads"], scale=1.0) - 2
            w[q + "left.o"], w[q + "left.o.b"], w[q + "left.out"] = rnd(W, a["heads"] * a["vdim"]), rnd(W, scale=0.1), gain(W)
            kd, vd = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            for n, rows in (("q", kd), ("k", kd), ("v", vd), ("g", vd), ("a1", lc["rank"])):
                w[q + "right." + n] = rnd(rows, W)
            w[q + "right.a2"], w[q + "right.a2.b"] = rnd(kd, lc["rank"], scale=1.0), rnd(kd, scale=1.0) + 1
            w[q + "right.norm"], w[q + "right.o"], w[q + "right.out"] = gain(r["vdim"]), rnd(W, vd), gain(W)
        f = lc["mlp"]
        if f is None:
            continue
        w[p + "norm2"] = gain(W)
        q = p + "mlp."
        n, ff = f["router"]["experts"], f["expert"]["ff"]
        w[q + "router"] = rnd(n, W, scale=2 * W**-0.5)
        up, down = rnd(ff, W), rnd(W, ff, scale=3 * ff**-0.5)
        for e in range(n):
            w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = rnd(ff, W), rnd(W, ff, scale=3 * ff**-0.5)
            if settled:       # experts so alike that a choice which rounding decides makes no difference to speak of
                w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = up + w[f"{q}e{e}.up"] * 0.1, down + w[f"{q}e{e}.down"] * 0.1
    return w


DESIGNS["Lotelix"] = (make_weights, oracle)
