"""Small Puzutar models for the tests: config dictionaries of several shapes, and random checkpoint tensors whose
attention is sharp, so that a key more or less in a window shows in the logits."""
import torch


def layer(heads, dim, rot, vdim, rank, window, ff, kv_from=None, base=1000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width, groups, vocab, side, eps=1e-5):
    return {"architecture": "Puzutar", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups},
            "token_side": {"dim": side}}


CONFIGS = {
    # layers that borrow another's rows, directly and across a layer in between
    "shared": config([layer(3, 24, 8, 16, 40, 37, 120), layer(3, 24, 8, 16, 40, 37, 120, kv_from=0),
                      layer(2, 16, 16, 24, 32, 21, 64), layer(4, 40, 8, 16, 40, 50, 48, kv_from=0)], 96, 3, 203, 12),
    # sizes that fit no vector or tile, layers of unequal sizes, one without a feed-forward
    "odd": config([layer(5, 20, 12, 24, 24, 5, 70), layer(2, 33, 6, 10, 50, 64, 0, base=77.0), layer(1, 8, 12, 7, 24, 200, 21, kv_from=0)],
                  100, 5, 131, 10),
    # one group, one head, one token of window
    "ones": config([layer(1, 16, 2, 8, 16, 1, 32), layer(1, 4, 4, 1, 1, 3, 1)], 48, 1, 97, 1),
    # more heads than one tile of rows, a latent of several column tiles
    "heads": config([layer(20, 40, 24, 40, 136, 150, 200), layer(20, 40, 24, 40, 136, 70, 200, kv_from=0)], 256, 4, 300, 24),
    "many": config([layer(70, 8, 8, 8, 32, 90, 96), layer(40, 16, 8, 16, 48, 33, 96)], 128, 2, 150, 8),
    # query heads too wide for the projected prefill, a latent wider than 256
    "tall": config([layer(2, 120, 16, 136, 272, 130, 160), layer(6, 64, 64, 32, 320, 100, 160)], 160, 4, 170, 16),
}


def tensors(cfg, seed=0, sharp=3.0):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    W, V, S = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    gain = lambda k: (1 + n(k, std=0.2).float()).to(torch.bfloat16)
    t = {"embed": n(V, W), "side.embed": n(V, len(cfg["layers"]) * S), "final.norm": gain(W)}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        t[p + "norm1"], t[p + "shift"] = gain(W), n(W, std=0.6)
        t[p + "mix.q"] = n(m["heads"] * (m["dim"] + m["rot_dim"]), W, std=sharp ** 0.5 * W ** -0.5)
        if m.get("kv_from") is None:
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = n(m["kv_rank"] + m["rot_dim"], W, std=sharp ** 0.5 * W ** -0.5), gain(m["kv_rank"])
        t[p + "mix.uk"] = n(m["heads"] * m["dim"], m["kv_rank"], std=m["kv_rank"] ** -0.5)
        t[p + "mix.uv"] = n(m["heads"] * m["vdim"], m["kv_rank"], std=m["kv_rank"] ** -0.5)
        t[p + "mix.o"] = n(W, m["heads"] * m["vdim"], std=1.5 * (m["heads"] * m["vdim"]) ** -0.5)
        if spec["mlp"]:
            f = spec["mlp"]["ff"]
            t[p + "mlp.up"], t[p + "mlp.up.b"], t[p + "mlp.act"] = n(f, W, std=W ** -0.5), n(f, std=0.3), n(2)
            t[p + "mlp.down"], t[p + "mlp.down.b"] = n(W, f, std=0.5 * f ** -0.5), n(W, std=0.1)
        t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = n(S, W, std=W ** -0.5), n(W, S), n(W, std=0.4)
    return t


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def write_checkpoint(path, cfg, t):
    import json
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.contiguous() for k, v in t.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(cfg))
    return path
