"""Plain restatement of the Pefitar decoder, one function per mechanism, whole sequence at a time.

Nothing here is fast and nothing is shared with the product path: every function takes the whole sequence
from position 0 and materialises whatever it needs (the full score matrix, the per-head keys and values of
the latent). ``dtype`` decides the precision; the tests run it in float64.

Notation: x [T, width] is the residual stream, h the normed input of a sublayer, p a prefix of tensor names.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis (eps inside the root), times a gain per channel."""
    return x * torch.rsqrt(x.square().mean(dim=-1, keepdim=True) + eps) * gain


def rotate(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, d]: coordinates 2i, 2i + 1 of the first ``dims`` turn by position * base^(-2i / dims)."""
    if dims == 0:
        return x
    T = x.shape[0]
    rate = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype, device=x.device)
    angle = torch.arange(T, dtype=x.dtype, device=x.device).reshape(T, 1, 1) * rate
    out = x.clone()
    even, odd = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = even * torch.cos(angle) - odd * torch.sin(angle)
    out[..., 1:dims:2] = odd * torch.cos(angle) + even * torch.sin(angle)
    return out


def visible(T: int, window=None) -> torch.Tensor:
    """Boolean [T, T]: position i sees j <= i, and with a window only the last ``window`` positions."""
    gap = torch.arange(T).reshape(T, 1) - torch.arange(T).reshape(1, T)
    see = gap >= 0
    return see if window is None else see & (gap < window)


def attend(q, k, v, scale, window=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; head h reads key / value head h // (H // G)."""
    T, H = q.shape[0], q.shape[1]
    per = H // k.shape[1]
    keys, vals = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    score = torch.einsum("ihd,jhd->hij", q, keys) * scale
    score = score.masked_fill(~visible(T, window).to(q.device), -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(score, dim=-1), vals)


def output_gate(out, h, w_gate):
    """Heads side by side [T, H * dv] times the logistic function of a projection of the mixer's input."""
    return out * torch.sigmoid(h @ w_gate.T)


def grouped_attention(h, w, p, spec):
    """Grouped-query causal attention with rotated queries and keys and a gated output."""
    T, H, G = h.shape[0], spec["heads"], spec["kv_heads"]
    base, dims = spec["rot"]["base"], spec["rot"]["dims"]
    q = rotate((h @ w[p + "q"].T).reshape(T, H, spec["dim"]), base, dims)
    k = rotate((h @ w[p + "k"].T).reshape(T, G, spec["dim"]), base, dims)
    v = (h @ w[p + "v"].T).reshape(T, G, spec["vdim"])
    out = attend(q, k, v, spec["scale"]).reshape(T, H * spec["vdim"])
    return output_gate(out, h, w[p + "g"]) @ w[p + "o"].T


def latent_queries(h, w, p, spec, eps):
    """[T, H, dim + rot_dim]: through a normed latent, the last rot_dim coordinates of every head rotated."""
    H, d, r = spec["heads"], spec["dim"], spec["rot_dim"]
    q = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    q = q.reshape(-1, H, d + r)
    return torch.cat([q[..., :d], rotate(q[..., d:], spec["rot"]["base"], spec["rot"]["dims"])], dim=-1)


def latent_cache(h, w, p, spec, eps):
    """What a position leaves behind: its normed latent [T, rank] and the rotated key part [T, rot_dim]."""
    n = spec["kv_rank"]
    down = h @ w[p + "dkv"].T
    turned = rotate(down[:, None, n:], spec["rot"]["base"], spec["rot"]["dims"])[:, 0]
    return rms_norm(down[:, :n], w[p + "dkv.norm"], eps), turned


def latent_attention(h, w, p, spec, eps):
    """Per-head keys and values from a shared latent, one rotated key part for all heads, a sliding window."""
    T, H, d, dv = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    q = latent_queries(h, w, p, spec, eps)
    c, turned = latent_cache(h, w, p, spec, eps)
    k = torch.cat([(c @ w[p + "uk"].T).reshape(T, H, d), turned[:, None].expand(T, H, -1)], dim=-1)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    return attend(q, k, v, spec["scale"], spec["mask"]["size"]).reshape(T, H * dv) @ w[p + "o"].T


def mixer(kind, h, w, p, spec, eps):
    return grouped_attention(h, w, p, spec) if kind == "attention" else latent_attention(h, w, p, spec, eps)


def dense_ff(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def sublayer(x, f, before, after, mult, eps):
    """The branch is normed on the way in and on the way out, and scaled before it joins the stream."""
    return x + mult * rms_norm(f(rms_norm(x, before, eps)), after, eps)


def order(config) -> list:
    """Layer numbers in the order they run: the looped range as often as it says, the others once."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    return [*range(loop["start"]), *list(range(loop["start"], loop["stop"])) * loop["times"], *range(loop["stop"], n)]


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(config: dict, weights: dict, tokens, dtype=torch.float64, layers_out=None, device="cpu"):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` (a list) receives the stream after each layer run."""
    w = {n: t.to(device=device, dtype=dtype) for n, t in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, device=device)]
    for i in order(config):
        spec, p = config["layers"][i], f"l{i}."
        x = sublayer(x, lambda h: mixer(spec["type"], h, w, p + "mix.", spec["mixer"], eps), w[p + "norm1"],
                     w[p + "norm1b"], m, eps)
        if spec["mlp"] is not None:
            x = sublayer(x, lambda h: dense_ff(h, w, p + "mlp."), w[p + "norm2"], w[p + "norm2b"], m, eps)
        if layers_out is not None:
            layers_out.append(x)
    return softcap(rms_norm(x, w["final.norm"], eps) @ w["embed"].T, config["logit_softcap"])
