"""Small Nipolorn models for the tests (own sizes, random weights)."""
import torch

from . import nipolorn_oracle as oracle
from .stack_helper import *  # noqa: F401,F403
from .stack_helper import DESIGNS


def mixer(heads=3, kv=1, dim=24, vdim=40, size=11, keep=3, scale=0.3, ssm_heads=6, ssm_vdim=20, state=12, groups=3, conv=3, norm_groups=5,
          left=0.8, right=1.3):
    return {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size, "keep_first": keep}},
            "right": {"heads": ssm_heads, "vdim": ssm_vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "left_scale": left, "right_scale": right}


def dense(ff=72, limit=0.9):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff=28, experts=5, top=2, shared=44):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width=88, vocab=101, eps=1e-5):
    return {"architecture": "Nipolorn", "layers": [{"type": "parallel", "mixer": m, "mlp": f} for m, f in layers],
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


#: unlike layers in one stack: head counts, head sizes, windows, states, feed-forward kinds, a layer without feed-forward
MIXED = config([(mixer(), dense()),
                (mixer(heads=4, kv=2, dim=64, vdim=64, size=70, keep=0, scale=0.125, ssm_heads=4, ssm_vdim=32, state=64, groups=1, conv=4,
                       norm_groups=1, left=1.1, right=0.4), moe()),
                (mixer(heads=8, kv=2, dim=96, vdim=128, size=33, keep=65, scale=0.1, ssm_heads=2, ssm_vdim=64, state=128, groups=2, conv=4,
                       norm_groups=2, left=0.5, right=0.7), None),
                (mixer(heads=5, kv=5, dim=33, vdim=7, size=1, keep=1, ssm_heads=3, ssm_vdim=17, state=9, groups=3, conv=1, norm_groups=3),
                 moe(ff=25, experts=9, top=3, shared=0))])
#: sizes that are no multiples of 8 anywhere
ODD = config([(mixer(heads=3, kv=3, dim=21, vdim=13, size=19, keep=5, ssm_heads=3, ssm_vdim=11, state=7, groups=1, conv=5, norm_groups=3),
               dense(ff=37, limit=2.5)), (mixer(), moe(ff=19, experts=3, top=1, shared=21))], width=75, vocab=67, eps=3e-6)
#: heads wider than the 16-bit kernels' tiles
WIDE = config([(mixer(heads=2, kv=1, dim=160, vdim=136, size=40, keep=4, scale=0.08), dense())], width=64, vocab=50)
#: everything a multiple of the tensor-core tiles: the fused prefill paths and the chunked scan run
TILED = config([(mixer(heads=8, kv=2, dim=128, vdim=128, size=150, keep=9, scale=0.09, ssm_heads=4, ssm_vdim=64, state=128, groups=2, conv=4,
                       norm_groups=2, left=1.2, right=0.9), dense(ff=192, limit=1.5)),
                (mixer(heads=4, kv=1, dim=64, vdim=64, size=300, keep=130, scale=0.125, ssm_heads=8, ssm_vdim=32, state=64, groups=1, conv=4,
                       norm_groups=4), moe(ff=64, experts=8, top=2, shared=128))], width=256, vocab=256)


def make_weights(cfg, seed, dtype, settled):
    """Random checkpoint tensors. Scales keep every branch audible in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, scale=None):
        return (torch.randn(shape, generator=g) * (shape[-1] ** -0.5 if scale is None else scale)).to(dtype)

    w = {"embed": rnd(V, W, scale=1.0), "final.norm": rnd(W, scale=0.2), "head": rnd(V, W)}
    for i, lc in enumerate(cfg["layers"]):
        p, a, r = f"l{i}.", lc["mixer"]["left"], lc["mixer"]["right"]
        inner, gn = r["heads"] * r["vdim"], r["groups"] * r["state"]
        for n in ("norm1", "norm1b", "norm2", "norm2b"):
            w[p + n] = rnd(W, scale=0.2)
        m = p + "mix.left."
        w[m + "q"], w[m + "k"] = rnd(a["heads"] * a["dim"], W), rnd(a["kv_heads"] * a["dim"], W)
        w[m + "v"], w[m + "o"] = rnd(a["kv_heads"] * a["vdim"], W), rnd(W, a["heads"] * a["vdim"])
        m = p + "mix.right."
        w[m + "in"] = rnd(2 * inner + 2 * gn + r["heads"], W)
        w[m + "conv"], w[m + "conv.b"] = rnd(inner + 2 * gn, r["conv"], scale=0.6), rnd(inner + 2 * gn, scale=0.2)
        w[m + "dt_bias"], w[m + "A_log"], w[m + "D"] = rnd(r["heads"], scale=1.0) - 2, rnd(r["heads"], scale=0.7), rnd(r["heads"], scale=1.0)
        w[m + "norm"], w[m + "o"] = 1 + rnd(inner, scale=0.2), rnd(W, inner)

        def glu(q, ff):
            w[q + "gate"], w[q + "up"], w[q + "down"] = rnd(ff, W), rnd(ff, W), rnd(W, ff)

        f = lc["mlp"]
        if f is None:
            del w[p + "norm2"], w[p + "norm2b"]
        elif f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
        else:
            for e in range(f["router"]["experts"]):
                glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
            w[p + "mlp.table"] = torch.stack([torch.randperm(f["router"]["experts"], generator=g)[:f["router"]["top"]]
                                              for _ in range(V)]).to(torch.int32)
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"])
    return w


DESIGNS["Nipolorn"] = (make_weights, oracle)
