"""Small Vulanex models for the tests: config dictionaries of several shapes, and random checkpoint tensors with sharp
attention, short and long memories and outputs whose sign no rounding turns."""
import json

import torch

YARN = {"factor": 4.0, "original": 60, "fast": 8.0, "slow": 1.0}


def attention(heads, kv, dim, coef=0.2, every=24, ff=0, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5}
    if every:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def par(heads, kv, dim, vdim, rot, size, pool, right, base=500.0, scaling=YARN, ff=0, scale=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.2 * dim ** -0.5, "mask": {"size": size, "pool": pool},
            "rot": {"dims": rot, "base": base}}
    if scaling:
        left["rot"]["scaling"] = scaling
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": right[0], "dim": right[1]}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None, "rank": right[2]}


def config(layers, width, vocab, taps, pair=(61, 7, 5), eps=1e-5, logit_scale=0.7):
    return {"architecture": "Vulanex", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps},
            "logit_scale": logit_scale, "embedding": {"bigram": {"buckets": pair[0], "mul_prev": pair[1], "mul_cur": pair[2]}}}


CONFIGS = {
    # groups of three query heads, key and value sizes that differ, blocks that straddle pages
    "mixed": config([par(6, 2, 40, 24, 24, 21, 6, (2, 24, 9), ff=72), attention(6, 2, 24, ff=56), par(4, 4, 24, 40, 24, 33, 12, (3, 40, 5), ff=40),
                     attention(4, 1, 32, 0.4, 7, ff=48)], 96, 203, 3),
    # sizes that fit no vector or tile, layers without a feed-forward, a long convolution, blocks of five
    "odd": config([attention(5, 1, 13, every=5), par(5, 1, 20, 33, 18, 7, 5, (3, 13, 3), scaling=None, ff=21), par(3, 3, 9, 7, 2, 11, 3, (1, 21, 1)),
                   attention(2, 2, 11, every=0, ff=19)], 100, 131, 6, (1, 1, 1)),
    # a window of one token beside blocks of one, one head, one pair row, two taps, a factor that grows with every position
    "ones": config([par(1, 1, 8, 8, 2, 1, 1, (1, 8, 1), ff=8), attention(1, 1, 8, 0.1, 1, ff=16), par(1, 1, 4, 8, 4, 2, 1, (1, 16, 2))], 48, 97, 2,
                   (2, 3, 1), logit_scale=1.0),
    # heads of 128, groups of four and eight, several key blocks and pieces
    "wide": config([par(8, 2, 128, 128, 64, 70, 16, (2, 128, 24), ff=160), attention(8, 1, 128, every=50, ff=96),
                    par(8, 1, 72, 96, 20, 45, 4, (1, 96, 300), ff=64)], 256, 300, 4, (997, 131, 17)),
    # shapes without a tensor-core attention kernel or pieces; blocks longer than a page; no history
    "tall": config([attention(20, 1, 24, ff=16), par(2, 1, 160, 200, 100, 50, 40, (1, 136, 8)), par(2, 2, 264, 300, 16, 20, 7, (2, 30, 4), ff=24),
                    attention(4, 2, 160, every=90)], 64, 150, 1),
    # one mixer only
    "plain": config([attention(4, 2, 32, ff=24), attention(2, 1, 48)], 64, 90, 3),
}


def tensors(cfg, seed=0, sharp=1.3):
    g = torch.Generator().manual_seed(seed)
    bf = torch.bfloat16
    n = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(bf)
    W, V = cfg["width"], cfg["vocab"]
    about = lambda k, c=1.0: (c + n(k, std=0.2 * c).float()).to(bf)
    lin = lambda o, i, gain=1.0: n(o, i, std=gain * i ** -0.5)
    t = {"embed": n(V, W), "bigram": n(cfg["embedding"]["bigram"]["buckets"] + 1, W, std=0.7), "final.norm": about(W), "final.norm.b": n(W, std=0.2)}
    for i, spec in enumerate(cfg["layers"]):
        m, p, f = spec["mixer"], f"l{i}.", spec["mlp"]
        x = p + "mix."
        for h in ("1", "2") if f else ("1",):
            t[p + "norm" + h], t[p + f"norm{h}.b"], t[p + "canon" + h] = about(W), n(W, std=0.2), n(W, cfg["canon"]["taps"], std=0.3)
        a = m if spec["type"] == "attention" else m["left"]
        y = x if spec["type"] == "attention" else x + "left."
        t[y + "q"], t[y + "k"], t[y + "o"] = lin(a["heads"] * a["dim"], W), lin(a["kv_heads"] * a["dim"], W), lin(W, a["heads"] * a["vdim"])
        if spec["type"] == "parallel":
            t[y + "v"], t[y + "sink"] = lin(a["kv_heads"] * a["vdim"], W), n(a["heads"])
            t[y + "q.norm"], t[y + "k.norm"] = about(a["dim"], sharp), about(a["dim"], sharp)
            H, d, rank, y = m["right"]["heads"], m["right"]["dim"], spec["rank"], x + "right."
            for k in ("k", "v", "g", "a"):
                t[y + k] = lin(H * d, W)
            # a token reads much of what it has just written: an output is no difference of numbers next to each other, whose
            # sign, which the norm makes of it, a rounding could turn
            t[y + "r"] = (0.8 * t[y + "k"].float() + 0.6 * lin(H * d, W).float()).to(bf)
            t[y + "a.b"], t[y + "w0"], t[y + "w1"], t[y + "w2"] = n(H * d), (2 * n(H * d).float() - 1).to(bf), lin(rank, W), lin(H * d, rank)
            t[y + "norm"], t[y + "o"] = about(H * d), lin(W, H * d)
            t[x + "left.out"], t[x + "right.out"] = about(W, 1.1), about(W, 0.9)
        if f:
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(f["ff"], W, 1.5), lin(f["ff"], W, 1.5), lin(W, f["ff"], 1.5)
    return t


def public(cfg):
    """The dictionary as a `config.json` has it."""
    return {**cfg, "layers": [{k: v for k, v in x.items() if k != "rank"} for x in cfg["layers"]]}


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def write_checkpoint(path, cfg, t):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.contiguous() for k, v in t.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(public(cfg)))
    return path
