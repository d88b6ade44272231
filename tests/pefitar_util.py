"""Small random Pefitar models for the tests: configurations and weights of a useful scale. None of the layer kinds,
counts or constants of one configuration repeats in another by need."""

import torch


def attention(heads=4, kv_heads=2, dim=16, vdim=24, dims=12, base=500.0, scale=0.3, ff=40):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "rot": {"base": base, "dims": dims}}}


def latent(heads=3, dim=10, rot_dim=6, vdim=14, q_rank=20, kv_rank=28, size=9, base=90.0, scale=0.25, ff=36):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "mask": {"size": size}, "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def config(layers=None, vocab=89, width=44, eps=2e-5, loop=(1, 3, 3), mult=0.7, cap=11.0):
    layers = layers or [latent(), attention(), latent(heads=5, size=17, vdim=8, kv_rank=12, q_rank=9, ff=None),
                        attention(heads=6, kv_heads=1, dim=14, dims=14, vdim=10, scale=0.4)]
    return {"architecture": "Pefitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "loop": dict(zip(("start", "stop", "times"), loop)), "residual_mult": mult, "logit_softcap": cap}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Weights that keep every branch of order one and every gain away from one."""
    gen = torch.Generator().manual_seed(seed)
    t = {}

    def draw(name, *shape, std=1.0, mean=0.0):
        t[name] = (torch.randn(shape, generator=gen) * std + mean).to(dtype)

    def mat(name, rows, cols, gain=1.0):
        draw(name, rows, cols, std=gain * cols ** -0.5)

    W = cfg["width"]
    draw("embed", cfg["vocab"], W)
    draw("final.norm", W, std=0.2, mean=1.2)
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if spec["mlp"] else ()):
            draw(p + n, W, std=0.3, mean=0.9)
        if spec["type"] == "attention":
            q, k, v, o = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
            for n, rows in (("q", q), ("k", k), ("v", v), ("g", o)):
                mat(f"{p}mix.{n}", rows, W, 1.5)
        else:
            H, d, r = m["heads"], m["dim"], m["rot_dim"]
            o = H * m["vdim"]
            mat(p + "mix.dq", m["q_rank"], W)
            draw(p + "mix.dq.norm", m["q_rank"], std=0.3, mean=1.2)
            mat(p + "mix.uq", H * (d + r), m["q_rank"], 1.5)
            mat(p + "mix.dkv", m["kv_rank"] + r, W)
            draw(p + "mix.dkv.norm", m["kv_rank"], std=0.3, mean=1.3)
            mat(p + "mix.uk", H * d, m["kv_rank"], 1.5)
            mat(p + "mix.uv", o, m["kv_rank"])
        mat(p + "mix.o", W, o)
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            mat(p + "mlp.gate", ff, W, 1.5)
            mat(p + "mlp.up", ff, W, 1.5)
            mat(p + "mlp.down", W, ff)
    return t
