"""Plain restatement of the Rorosun decoder, one function per mechanism, whole sequence at a time.

Nothing here is fast and nothing is shared with the product path: every function takes the whole
sequence from position 0 and materialises whatever it needs (the full score matrix, one recurrent
state after another). ``dtype`` of the inputs decides the precision; the tests run it in float64.

Notation: x [T, width] is the residual stream, h the normed input of a branch.
"""

from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms(x, eps) * gain.reshape(())


def visible(T: int, size: int, pool: int):
    """Boolean masks [T, T] (tokens) and [T, T // pool] (pooled blocks) of what each position sees."""
    i = torch.arange(T).reshape(-1, 1)
    j = torch.arange(T).reshape(1, -1)
    tokens = (j <= i) & (i - j < size)
    last = torch.arange(T // pool).reshape(1, -1) * pool + pool - 1
    return tokens, last <= i - size


def pool_blocks(x: torch.Tensor, pool: int) -> torch.Tensor:
    """Means over the complete blocks of ``pool`` rows: [T, ...] -> [T // pool, ...]."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(1)


def window_pool_weights(q, k, scale, size, pool):
    """q [T, H, d], k [T, G, d] -> softmax weights [H, T, T + T // pool] over tokens and pooled blocks."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    keys = torch.cat([k, pool_blocks(k, pool)]).repeat_interleave(per, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, keys) * scale
    mask = torch.cat(visible(T, size, pool), dim=1).to(q.device)
    return torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1)


def talk(weights, mix):
    """Each head's weights become a linear combination of all heads' weights."""
    return torch.einsum("hg,gij->hij", mix, weights)


def apply_values(weights, v, pool):
    """weights [H, T, T + blocks], v [T, G, dv] -> [T, H, dv]."""
    per = weights.shape[0] // v.shape[1]
    vals = torch.cat([v, pool_blocks(v, pool)]).repeat_interleave(per, dim=1)
    return torch.einsum("hij,jhd->ihd", weights, vals)


def left_mixer(h, w, p, spec, eps):
    """Window + pooled-block attention with normed q / k and mixed heads."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    q = (rms(q, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (rms(k, eps) * w[p + "k.norm"]).reshape(T, G, d)
    size, pool = spec["mask"]["size"], spec["mask"]["pool"]
    a = talk(window_pool_weights(q, k, spec["scale"], size, pool), w[p + "talk"])
    return apply_values(a, v.reshape(T, G, dv), pool).reshape(T, H * dv) @ w[p + "o"].T


def shift_mix(h, mu):
    """h + (previous token's h - h) * mu, zeros before the first token."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def decay(mix_w, w1, w2, w0):
    return torch.exp(-torch.exp(torch.tanh(mix_w @ w1.T) @ w2.T + w0))


def wkv(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, d]; u [H, d]; state [H, key, value]. Returns o [T, H, d] and the last state."""
    T, H, d = r.shape
    S = torch.zeros(H, d, d, dtype=r.dtype, device=r.device) if state is None else state
    out = []
    for t in range(T):
        kv = k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(torch.einsum("hkv,hk->hv", S + u.unsqueeze(-1) * kv, r[t]))
        S = w[t].unsqueeze(-1) * S + kv
    return torch.stack(out), S


def right_mixer(h, w, p, spec, eps):
    """Time mixing with a matrix state per head."""
    T, H, d = h.shape[0], spec["heads"], spec["dim"]
    mix = {s: shift_mix(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).reshape(T, H, d) for s in "rkv")
    gate = mix["g"] @ w[p + "g"].T
    gate = gate * torch.sigmoid(gate)
    dec = decay(mix["w"], w[p + "w1"], w[p + "w2"], w[p + "w0"]).reshape(T, H, d)
    o, _ = wkv(r, k, v, dec, w[p + "u"])
    return (rms(o, eps).reshape(T, H * d) * w[p + "norm"] * gate) @ w[p + "o"].T


def parallel_mixer(h, w, p, spec, eps):
    return spec["left_scale"] * left_mixer(h, w, p + "left.", spec["left"], eps) + \
        spec["right_scale"] * right_mixer(h, w, p + "right.", spec["right"], eps)


def dense_ff(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(config: dict, weights: dict, tokens, dtype=torch.float64, layers_out=None, device="cpu"):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` (a list) receives the stream after each layer."""
    w = {n: t.to(device=device, dtype=dtype) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, device=device)]
    for i, spec in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + parallel_mixer(scalar_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps) * w[p + "ls1"]
        if spec["mlp"] is not None:
            x = x + dense_ff(scalar_norm(x, w[p + "norm2"], eps), w, p + "mlp.") * w[p + "ls2"]
        if layers_out is not None:
            layers_out.append(x)
    return scalar_norm(x, w["final.norm"], eps) @ w["head"].T
