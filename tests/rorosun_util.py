"""Small random Rorosun models for the tests: configurations, weights of a useful scale, model folders."""

import json
import os
import struct

import torch


def layer(heads=4, kv_heads=2, dim=16, vdim=24, size=10, pool=3, scale=0.3, left_scale=0.8, right_scale=0.6,
          r_heads=3, r_dim=20, ff=40):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                               "mask": {"size": size, "pool": pool}},
                      "right": {"heads": r_heads, "dim": r_dim},
                      "left_scale": left_scale, "right_scale": right_scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers=None, vocab=97, width=48, eps=1e-5):
    return {"architecture": "Rorosun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": layers or [layer(), layer(size=7, pool=4, ff=None, kv_heads=4, r_dim=8, scale=0.5),
                                 layer(heads=6, kv_heads=3, dim=10, vdim=6, size=5, pool=8, left_scale=-0.4, ff=56)]}


def weights(cfg, seed=0, rank=5, dtype=torch.bfloat16):
    """Weights that keep every branch of order one; every vector that a model could happen to hold as all
    ones, zeros or an identity is drawn at random."""
    gen = torch.Generator().manual_seed(seed)
    t = {}

    def draw(name, *shape, std=1.0, mean=0.0):
        t[name] = (torch.randn(shape, generator=gen) * std + mean).to(dtype)

    def mat(name, rows, cols, gain=1.0):
        draw(name, rows, cols, std=gain * cols ** -0.5)

    W, V = cfg["width"], cfg["vocab"]
    draw("embed", V, W)
    mat("head", V, W)
    draw("final.norm", std=0.1, mean=1.3)
    for i, spec in enumerate(cfg["layers"]):
        p, l, r = f"l{i}.", spec["mixer"]["left"], spec["mixer"]["right"]
        q, k, v, N = l["heads"] * l["dim"], l["kv_heads"] * l["dim"], l["kv_heads"] * l["vdim"], r["heads"] * r["dim"]
        draw(p + "norm1", std=0.1, mean=0.8)
        for n, rows in (("q", q), ("k", k), ("v", v)):
            mat(f"{p}mix.left.{n}", rows, W)
            draw(f"{p}mix.left.{n}.b", rows, std=0.5)
        draw(p + "mix.left.q.norm", q, std=0.3, mean=1.5)
        draw(p + "mix.left.k.norm", k, std=0.3, mean=1.2)
        draw(p + "mix.left.talk", l["heads"], l["heads"], std=0.6)
        mat(p + "mix.left.o", W, l["heads"] * l["vdim"])
        for s in "rkvgw":
            draw(f"{p}mix.right.mu.{s}", W, std=0.3, mean=0.5)
        for s in "rkvg":
            mat(f"{p}mix.right.{s}", N, W)
        mat(p + "mix.right.w1", rank, W)
        mat(p + "mix.right.w2", N, rank)
        draw(p + "mix.right.w0", N, std=1.0, mean=-2.0)
        draw(p + "mix.right.u", r["heads"], r["dim"], std=0.7)
        draw(p + "mix.right.norm", N, std=0.3, mean=1.0)
        mat(p + "mix.right.o", W, N)
        draw(p + "ls1", W, std=0.3, mean=0.7)
        if spec["mlp"] is not None:
            ff = spec["mlp"]["ff"]
            draw(p + "norm2", std=0.1, mean=1.1)
            mat(p + "mlp.gate", ff, W)
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
            draw(p + "ls2", W, std=0.3, mean=0.6)
    return t


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_NAMES = {torch.bfloat16: "BF16", torch.float32: "F32", torch.float16: "F16"}


def write_safetensors(path, tensors):
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": _NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def write_model(folder, cfg, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return str(folder)


def rel(a, b):
    """Largest row error: root mean square of the difference over that of the expected values."""
    a, b = torch.as_tensor(a).double().cpu(), torch.as_tensor(b).double().cpu()
    return float(((a - b).pow(2).mean(-1).sqrt() / b.pow(2).mean(-1).sqrt().clamp_min(1e-30)).max())
