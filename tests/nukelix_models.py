"""Small Nukelix models for the tests: config dictionaries of several shapes, and random checkpoint tensors with sharp
attention, long and short memories and experts whose choice no rounding turns."""
import json

import torch

WAVES = {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 48}
YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def attention(heads, kv, dim, vdim, rot, window=None, keep=0, mix=True, base=300.0, scaling=None, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "rot": {"dims": rot, "base": base}}
    if scaling:
        m["rot"]["scaling"] = scaling
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": mlp}


def par(heads, kv, dim, vdim, rot, right, cap=12.0, base=2000.0, mlp=None, scales=(1.1, 0.7)):
    left = attention(heads, kv, dim, vdim, rot, mix=False, base=base)["mixer"]
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "left_scale": scales[0], "right_scale": scales[1], "right": {
        "heads": right[0], "dim": right[1], "vdim": right[2], "gate_cap": cap}}}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, rot_dims=None, base=700.0, scaling=YARN, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": 1.4 * (dim + rot) ** -0.5,
         "rot": {"dims": rot_dims or rot, "base": base}}
    if scaling:
        m["rot"]["scaling"] = scaling
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, shared=0):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {**d, "shared": {"ff": shared}} if shared else d


def config(layers, width, vocab, eps=1e-5, cap=20.0):
    return {"architecture": "Nukelix", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap}


CONFIGS = {
    # groups of three query heads, key and value sizes that differ, windows that differ, partial rotation, several mixed values
    "mixed": config([par(6, 2, 40, 24, 24, (2, 16, 24), mlp=moe(5, 3, 40, 56)),
                     attention(6, 2, 24, 32, 12, 37, 5, scaling=WAVES, mlp=moe(4, 2, 24, 40)),
                     latent(5, 24, 8, 16, 36, 40, mlp=moe(6, 1, 32, 24)), attention(4, 2, 40, 32, 40, 20, 18, mlp=moe(3, 3, 24)),
                     attention(4, 4, 16, 24, 8, 50, 1, mix=False, scaling=WAVES), par(4, 4, 24, 40, 24, (3, 40, 16), 5.0, mlp=moe(4, 2, 48, 16))],
                    96, 203),
    # sizes that fit no vector or tile, layers without a feed-forward, latent attention first, one expert per token
    "odd": config([latent(3, 13, 6, 11, 21, 19, rot_dims=4, mlp=moe(3, 1, 21, 13)), par(5, 1, 20, 33, 18, (3, 13, 7)),
                   attention(5, 1, 21, 7, 10, 6, 3, scaling=WAVES, mlp=moe(7, 2, 10, 9)), attention(1, 1, 9, 7, 2, 33, 0, base=50.0),
                   latent(1, 7, 2, 5, 9, 50, scaling=None, mlp=moe(2, 2, 8))], 100, 131),
    # a window of one token beside one kept token, one head, one expert
    "ones": config([attention(1, 1, 4, 8, 4, 1, 1, mlp=moe(1, 1, 8, 8)), par(1, 1, 4, 8, 2, (1, 8, 8), 3.0, mlp=moe(2, 1, 8)),
                    attention(1, 1, 16, 8, 8, 3, 0, mlp=moe(1, 1, 9, 16)), latent(1, 8, 2, 8, 8, 16)], 48, 97),
    # heads of 128, groups of four and eight, several pieces and key blocks, more kept tokens than a key block holds
    "wide": config([par(8, 2, 128, 128, 64, (2, 96, 128), 15.0, mlp=moe(6, 2, 64, 96)), latent(4, 96, 32, 128, 104, 240, mlp=moe(4, 4, 32, 40)),
                    attention(8, 1, 128, 96, 128, 70, 75, scaling=WAVES, mlp=moe(3, 1, 40)), attention(8, 1, 72, 96, 20, 150, 3)], 256, 300),
    # shapes without a tensor-core attention kernel or chunked form
    "tall": config([attention(20, 1, 24, 24, 8, 40, 6, mix=False, mlp=moe(2, 1, 16)), par(2, 1, 160, 200, 100, (1, 272, 24)),
                    latent(33, 130, 20, 24, 40, 300), attention(2, 2, 264, 300, 16, 90, 2, mlp=moe(3, 2, 16, 24))], 64, 150),
    # nothing recurrent; attention that sees everything
    "stateless": config([attention(4, 2, 32, 32, 16, mix=False, mlp=moe(3, 1, 24)), latent(2, 16, 8, 24, 24, 32)], 64, 90),
}


def tensors(cfg, seed=0, sharp=1.3):
    g = torch.Generator().manual_seed(seed)
    bf = torch.bfloat16
    n = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(bf)
    W, V = cfg["width"], cfg["vocab"]
    about = lambda k, c=1.0: (c + n(k, std=0.2 * c).float()).to(bf)
    lin = lambda o, i, gain=1.0: n(o, i, std=gain * i ** -0.5)
    # The first E numbers of the stream stay close to the embedding's, levels half apart in a random order, and are what the
    # routers mostly read: no rounding turns the choice of experts.
    E = max((s["mlp"]["router"]["experts"] for s in cfg["layers"] if s["mlp"]), default=0)
    embed = n(V, W)
    for t in range(V):
        embed[t, :E] = (0.5 * torch.randperm(E, generator=g).float() - 0.25 * E).to(bf)

    def out_norm():
        w = about(W, 0.7)
        w[:E] = 0.01
        return w
    t = {"embed": embed, "final.norm": about(W)}

    def grouped(p, m):
        nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        for k, rows in (("q", nq), ("k", nk), ("v", nv)):
            t[p + k], t[p + k + ".b"] = lin(rows, W), n(rows, std=0.3)
        t[p + "q.norm"], t[p + "k.norm"], t[p + "g"], t[p + "o"] = about(nq, sharp), about(nk), lin(m["heads"], W), lin(W, m["heads"] * m["vdim"])

    for i, spec in enumerate(cfg["layers"]):
        m, p, f = spec["mixer"], f"l{i}.", spec["mlp"]
        x = p + "mix."
        t[p + "norm1"] = out_norm()
        if f:
            t[p + "norm2"] = out_norm()
        if spec["type"] == "attention":
            grouped(x, m)
            if m.get("v_mix"):
                t[x + "vmix"] = (0.35 + 0.1 * i + n(1, std=0.05).float()).to(bf)[0]
        elif spec["type"] == "latent_attention":
            H, r = m["heads"], m["kv_rank"]
            t[x + "dq"], t[x + "dq.norm"] = lin(m["q_rank"], W), about(m["q_rank"], sharp)
            t[x + "uq"] = lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            t[x + "dkv"], t[x + "dkv.norm"] = lin(r + m["rot_dim"], W), about(r)
            t[x + "uk"], t[x + "uv"], t[x + "g"], t[x + "o"] = lin(H * m["dim"], r), lin(H * m["vdim"], r), lin(H, W), lin(W, H * m["vdim"])
        else:
            grouped(x + "left.", m["left"])
            b, y = m["right"], x + "right."
            H = b["heads"]
            for k, rows in (("q", H * b["dim"]), ("k", H * b["dim"]), ("v", H * b["vdim"]), ("g", H * b["vdim"])):
                t[y + k] = lin(rows, W)
            # a key and its own query point the same way: an output is no difference of numbers next to each other, whose
            # sign, which the norm makes of it, a rounding could turn
            t[y + "k"] = (0.8 * t[y + "q"].float() + 0.6 * t[y + "k"].float()).to(bf)
            t[y + "norm"], t[y + "o"] = about(H * b["vdim"]), lin(W, H * b["vdim"])
            t[y + "i"], t[y + "i.b"], t[y + "f"], t[y + "f.b"] = lin(H, W, 1.5), n(H), lin(H, W), (3.0 + 1.5 * n(H).float()).to(bf)
        if f:
            ff = f["expert"]["ff"]
            for e, k in [(f"e{e}", ff) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if "shared" in f else []):
                for name, shape in (("gate", (k, W)), ("up", (k, W)), ("down", (W, k))):
                    t[p + f"mlp.{e}.{name}"] = lin(*shape, 1.5)
            router = n(f["router"]["experts"], W, std=0.005)
            router[:, :router.shape[0]] += 1.2 * torch.eye(router.shape[0]).to(bf)
            t[p + "mlp.router"] = router
    return t


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def write_checkpoint(path, cfg, t):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.contiguous() for k, v in t.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(cfg))
    return path
