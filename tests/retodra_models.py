"""Small Retodra models for the tests: config dictionaries of several shapes, and random checkpoint tensors with sharp
attention, long and short memories, so that one key more or less in a window or a lost state shows in the logits."""
import json
import math

import torch


def gla(heads, dim, vdim, tau=8.0, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def par(heads, kv, dim, vdim, window, far, right, mlp=None, cap=8.0, scale=None, scales=(0.9, 0.55)):
    rh, rd, rv = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale or dim ** -0.5,
                 "softcap": cap, "bias_max": far},
        "right": {"heads": rh, "dim": rd, "vdim": rv, "decay": [math.exp(-2.0 ** -(7.0 * (h + 1) / rh)) for h in range(rh)]},
        "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}


def config(layers, width, vocab, eps=1e-5, scale=None):
    return {"architecture": "Retodra", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": scale or width ** 0.5}}


CONFIGS = {
    # groups of three query heads, key and value sizes that differ, windows that differ from layer to layer
    "mixed": config([gla(3, 24, 40, mlp=dense(120)), par(6, 2, 40, 24, 37, 90, (2, 16, 24), moe(5, 3, 3, 40)),
                     gla(2, 48, 24, 3.0, dense(72)), par(4, 4, 24, 48, 70, 150, (5, 24, 8), moe(4, 1, 2, 24))], 96, 203),
    # sizes that fit no vector or tile, a layer without a feed-forward, attention first, no identity experts
    "odd": config([par(5, 1, 20, 33, 5, 40, (3, 13, 7), moe(3, 0, 1, 21)), gla(1, 18, 33, 1.0), par(2, 2, 66, 5, 200, 300, (1, 9, 50), None),
                   gla(5, 7, 11, 30.0, moe(2, 5, 4, 10))], 100, 131),
    # a window of one token, one head, one expert, keys of one number; experts on linear layers and dense parallel ones.
    # (Values of one number are left to the tests of the ops: normed, they are nothing but a sign.)
    "ones": config([par(1, 1, 4, 8, 1, 90, (1, 1, 8), dense(16)), gla(1, 1, 16, 1.0, moe(1, 1, 2, 8)),
                    par(1, 1, 16, 8, 3, 90, (1, 8, 8), moe(1, 0, 1, 9))], 48, 97, scale=1.0),
    # heads of 128, groups of four and eight, several pieces and key blocks; strong channel decays
    "wide": config([gla(2, 96, 128, 1.0, dense(200)), par(8, 2, 128, 128, 150, 400, (2, 64, 96), moe(6, 2, 2, 64)),
                    par(8, 1, 72, 100, 70, 150, (2, 128, 32), None)], 256, 300),
    # shapes without a tensor-core attention kernel or chunked form: heads beyond 128 with large groups, keys beyond 256
    "tall": config([par(16, 1, 136, 40, 33, 80, (1, 272, 24), dense(64)), par(20, 1, 24, 24, 90, 200, (1, 16, 260), None), gla(1, 288, 40, 4.0),
                    par(2, 1, 160, 256, 64, 130, (1, 8, 8), None)], 64, 150),
    # no attention at all
    "linear": config([gla(2, 32, 64, 16.0, dense(48)), gla(4, 16, 16, 2.0, moe(4, 4, 2, 32))], 80, 111),
}


def ranks(i):
    return (6, 16, 1, 9)[i % 4]


def buckets(i):
    return (12, 8, 32, 2)[i % 4]


def tensors(cfg, seed=0, sharp=2.5, step=0.2):
    """`step`: distance between the routers' corrections. 1.0 fixes the choice of experts (no rounding turns it), less lets
    the scores decide."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    W, V = cfg["width"], cfg["vocab"]
    near = lambda k: n(k, std=0.2)
    about = lambda k, c=1.0: (c + n(k, std=0.2 * c).float()).to(torch.bfloat16)
    lin = lambda o, i, gain=1.0: n(o, i, std=gain * i ** -0.5)
    t = {"embed": n(V, W, std=1 / cfg["embedding"]["scale"]), "head": lin(V, W), "final.norm": near(W)}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        for h in ("1", "2") if spec["mlp"] else ("1",):
            t[p + "norm" + h], t[p + f"norm{h}b"], t[p + "ls" + h] = near(W), near(W), about(W, 0.6)
        if spec["type"] == "gla":
            H, K, E, r = m["heads"], m["dim"], m["vdim"], ranks(i)
            for k, rows in (("q", H * K), ("k", H * K), ("v", H * E), ("g", H * E), ("a1", r)):
                t[p + "mix." + k] = lin(rows, W)
            t[p + "mix.a2"], t[p + "mix.a2.b"] = n(H * K, r, std=1.5 * r ** -0.5), (1.5 + n(H * K, std=1.5).float()).to(torch.bfloat16)
            t[p + "mix.norm"], t[p + "mix.o"] = about(E), lin(W, H * E)
        else:
            a, b = m["left"], m["right"]
            nq, nk, nv = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            for k, rows in (("q", nq), ("k", nk), ("v", nv), ("g", a["heads"] * a["vdim"])):
                t[p + "mix.left." + k] = lin(rows, W)
            t[p + "mix.left.q.norm"], t[p + "mix.left.k.norm"] = about(nq, sharp), about(nk)
            t[p + "mix.left.rel"], t[p + "mix.left.o"] = n(buckets(i), a["heads"], std=1.2), lin(W, a["heads"] * a["vdim"])
            for k, rows in (("q", b["heads"] * b["dim"]), ("k", b["heads"] * b["dim"]), ("v", b["heads"] * b["vdim"]), ("g", b["heads"] * b["vdim"])):
                t[p + "mix.right." + k] = lin(rows, W, 1.5)
            t[p + "mix.right.norm"], t[p + "mix.right.o"] = about(b["heads"] * b["vdim"]), lin(W, b["heads"] * b["vdim"])
        f = spec["mlp"]
        if f and f["kind"] == "dense":
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"])
        elif f:
            ff, r = f["expert"]["ff"], f["router"]
            for e in range(r["experts"]):
                t[p + f"mlp.e{e}.gate"], t[p + f"mlp.e{e}.up"], t[p + f"mlp.e{e}.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
            outs = r["experts"] + r["identity"]
            t[p + "mlp.router"], t[p + "mlp.correction"] = lin(outs, W, 2.0), (step * torch.randperm(outs, generator=g)).to(torch.bfloat16)
    return t


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def write_checkpoint(path, cfg, t):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.contiguous() for k, v in t.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(cfg))
    return path
