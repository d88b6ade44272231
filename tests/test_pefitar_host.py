"""Pefitar without a GPU: the plain implementation's own properties, configuration and checkpoint reading, the
order of layer runs, the sequence state and the C ABI of the causal attention kernels."""

import copy
import ctypes
import json
import math
import os
import shutil
import subprocess

import pytest
import torch

from conftest import ROOT
from leankv_b200 import _native, registry
from leankv_b200.mixer_engine import MixerDecodeEngine, MixerModelConfig
from leankv_b200.mixers import AttentionSpec, LatentSpec, Rotation, _per_head_padded
from leankv_b200.sequence_state import SequenceState
from oracle import pefitar as plain
from pefitar_util import attention, config, latent, weights
from rorosun_util import tokens, write_model

F64 = torch.float64


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


# ── the plain implementation ─────────────────────────────────────────────────────────────────

def test_rotation_turns_neighbouring_pairs_and_keeps_the_rest():
    x = torch.randn(9, 2, 10, generator=gen(), dtype=F64)
    y = plain.rotate(x, 50.0, 6)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    for p in range(9):
        for i in range(3):
            a = p * 50.0 ** (-2 * i / 6)
            z = complex(x[p, 1, 2 * i], x[p, 1, 2 * i + 1]) * complex(math.cos(a), math.sin(a))
            assert abs(complex(y[p, 1, 2 * i], y[p, 1, 2 * i + 1]) - z) < 1e-12


def test_rotated_scores_depend_on_the_distance_only():
    q, k = (torch.randn(8, generator=gen(s), dtype=F64).expand(30, 1, 8) for s in (1, 2))
    s = torch.einsum("ihd,jhd->ij", plain.rotate(q, 100.0, 8), plain.rotate(k, 100.0, 8))
    for gap in (-3, 0, 1, 7):
        d = torch.diagonal(s, offset=gap)
        assert torch.allclose(d, d[0].expand_as(d))


def test_visibility_by_enumeration():
    for window in (None, 1, 4, 7, 100):
        see = plain.visible(20, window)
        for i in range(20):
            assert see[i].nonzero().flatten().tolist() == [j for j in range(20) if j <= i and (window is None or i - j < window)]


def test_attention_against_a_loop():
    T, H, G, d, dv = 6, 4, 2, 3, 5
    q, k, v = (torch.randn(T, n, w, generator=gen(s), dtype=F64) for s, n, w in ((1, H, d), (2, G, d), (3, G, dv)))
    out = plain.attend(q, k, v, 0.7, 3)
    for i in range(T):
        for h in range(H):
            js = [j for j in range(max(0, i - 2), i + 1)]
            e = [math.exp(0.7 * float(q[i, h] @ k[j, h // 2])) for j in js]
            want = sum(x / sum(e) * v[j, h // 2] for x, j in zip(e, js))
            assert torch.allclose(out[i, h], want)


def test_latent_scores_equal_folded_queries_against_latents():
    """(W c) . q is c . (W^T q), and a mean of W c is W times the mean: what a decode step relies on."""
    cfg = config()
    spec, p = cfg["layers"][0]["mixer"], "l0.mix."
    w = {n: t.double() for n, t in weights(cfg).items()}
    h = torch.randn(12, cfg["width"], generator=gen(), dtype=F64)
    q = plain.latent_queries(h, w, p, spec, 1e-5)
    c, turned = plain.latent_cache(h, w, p, spec, 1e-5)
    H, d, n = spec["heads"], spec["dim"], spec["kv_rank"]
    folded = torch.einsum("thd,hdn->thn", q[..., :d], w[p + "uk"].reshape(H, d, n))
    keys = torch.cat([c, turned], -1)[:, None]
    mean = plain.attend(torch.cat([folded, q[..., d:]], -1), keys, c[:, None], spec["scale"], spec["mask"]["size"])
    out = torch.einsum("thn,hvn->thv", mean, w[p + "uv"].reshape(H, -1, n)).reshape(12, -1) @ w[p + "o"].T
    assert torch.allclose(out, plain.latent_attention(h, w, p, spec, 1e-5))


def test_order_of_layer_runs():
    c = config(loop=(1, 3, 3))
    assert plain.order(c) == [0, 1, 2, 1, 2, 1, 2, 3] == MixerModelConfig.from_dict(c).order
    for loop, want in (((0, 4, 1), [0, 1, 2, 3]), ((2, 2, 5), [0, 1, 2, 3]), ((3, 4, 2), [0, 1, 2, 3, 3]),
                       ((0, 1, 2), [0, 0, 1, 2, 3])):
        c = config(loop=loop)
        assert plain.order(c) == want == MixerModelConfig.from_dict(c).order
    del c["loop"]
    assert plain.order(c) == [0, 1, 2, 3] == MixerModelConfig.from_dict(c).order


def test_plain_model_is_causal_and_every_parameter_matters():
    cfg = config()
    w, ids = weights(cfg), tokens(cfg, 24)
    full = plain.forward(cfg, w, ids)
    assert torch.allclose(plain.forward(cfg, w, ids[:17]), full[:17])
    assert float(full.abs().max()) < cfg["logit_softcap"]
    for name in w:
        ch = {n: t.float() * (1.25 if n == name else 1.0) + (0.1 if n == name else 0.0) for n, t in w.items()}
        assert not torch.allclose(plain.forward(cfg, ch, ids), full, atol=1e-6), f"{name} has no effect"


def _changes():
    yield "eps", lambda c: c["norm"].update(eps=0.1)
    yield "residual_mult", lambda c: c.update(residual_mult=0.9)
    yield "logit_softcap", lambda c: c.update(logit_softcap=7.0)
    yield "loop", lambda c: c["loop"].update(times=2)
    for layer, key, value in ((1, "scale", 0.5), (0, "scale", 0.5)):
        yield f"{layer}.{key}", lambda c, l=layer, k=key, v=value: c["layers"][l]["mixer"].update({k: v})
    yield "window", lambda c: c["layers"][0]["mixer"]["mask"].update(size=8)
    for layer in (0, 1):
        yield f"{layer}.base", lambda c, l=layer: c["layers"][l]["mixer"]["rot"].update(base=33.0)
    yield "dims", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10)


@pytest.mark.parametrize("what,change", list(_changes()), ids=[n for n, _ in _changes()])
def test_plain_model_reads_every_constant(what, change):
    cfg = config()
    w, ids = weights(cfg), tokens(cfg, 24)
    other = copy.deepcopy(cfg)
    change(other)
    assert not torch.allclose(plain.forward(other, w, ids), plain.forward(cfg, w, ids), atol=1e-6)


# ── configuration, registry, state ───────────────────────────────────────────────────────────

def test_config_reading():
    c = json.loads(json.dumps(config(vocab=31, width=24, eps=3e-4, loop=(0, 2, 2), mult=0.25, cap=9.0)))
    m = MixerModelConfig.from_dict(c)
    assert (m.vocab_size, m.hidden_size, m.eps, len(m.layers), m.loop, m.residual_mult, m.logit_softcap) == \
        (31, 24, 3e-4, 4, (0, 2, 2), 0.25, 9.0)
    for change in (lambda d: d.update(extra=1), lambda d: d["norm"].update(offset=1),
                   lambda d: d["layers"][0].update(type="parallel"), lambda d: d["layers"][0].update(gate=1),
                   lambda d: d["loop"].update(stop=9), lambda d: d["loop"].update(times=0), lambda d: d["loop"].update(more=1)):
        bad = copy.deepcopy(c)
        change(bad)
        with pytest.raises(ValueError):
            MixerModelConfig.from_dict(bad)
    c["logit_softcap"] = None
    assert MixerModelConfig.from_dict(c).logit_softcap == 0.0


def test_mixer_settings():
    s = AttentionSpec.from_dict(attention(heads=6, kv_heads=2, dim=20, vdim=8, dims=4, base=3.0, scale=0.5)["mixer"])
    assert s == AttentionSpec(6, 2, 20, 8, 0.5, Rotation(3.0, 4), None)
    l = LatentSpec.from_dict(latent(size=33)["mixer"])
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.size) == (3, 10, 6, 14, 20, 28, 33)
    good = attention()["mixer"]
    for change in ({"kv_heads": 3}, {"dim": 0}, {"rot": {"base": 9.0, "dims": 18}}, {"rot": {"base": 9.0, "dims": 3}},
                   {"rot": {"base": 9.0, "dims": 2, "more": 1}}, {"mask": {"size": 0}}, {"mask": {"size": 3, "pool": 2}}):
        with pytest.raises(ValueError):
            AttentionSpec.from_dict({**good, **change})
    with pytest.raises(TypeError):
        AttentionSpec.from_dict({**good, "bias": True})
    with pytest.raises(ValueError):
        LatentSpec.from_dict({**latent()["mixer"], "kv_rank": 0})


def test_rotation_rates():
    r = Rotation(10000.0, 8).rate("cpu")
    assert r.dtype == torch.float32 and torch.allclose(r.double(), torch.tensor([1.0, 0.1, 0.01, 0.001], dtype=F64))


def test_heads_are_padded_with_zero_rows():
    w = torch.randn(3 * 10, 4, generator=gen())
    p = _per_head_padded(w, 3, 10).reshape(3, 16, 4)
    assert torch.equal(p[:, :10].reshape(30, 4), w) and float(p[:, 10:].abs().max()) == 0.0
    assert torch.equal(_per_head_padded(torch.ones(32, 4), 2, 16), torch.ones(32, 4))


def test_registry_serves_the_design(tmp_path):
    assert "Pefitar" in registry.architectures()
    assert registry.supports({"architecture": "Pefitar"}, "float32") and registry.supports({"architecture": "Pefitar"}, "bfloat16")
    folder = write_model(tmp_path / "m", config(), weights(config()))
    with pytest.raises(ValueError, match="float16"):
        registry.load_engine(folder, dtype="float16")


def test_random_tensors_have_the_checkpoints_names_and_shapes():
    cfg = config()
    want = {n: t.shape for n, t in weights(cfg).items()}
    got = MixerDecodeEngine.random_tensors(MixerModelConfig.from_dict(cfg), "cpu")
    assert {n: t.shape for n, t in got.items()} == want and all(t.dtype == torch.bfloat16 for t in got.values())


def test_causal_state_sizes():
    seq = SequenceState("cpu", torch.bfloat16, max_seq_len=1000, max_chunk=64)
    full = seq.causal(kv_heads=2, dim=20, vdim=40, shared=0, size=1000)
    assert full.k.shape == (1024, 2, 32) and full.v.shape == (1024, 2, 48) and full.shared is None and full.ring == 1024
    window = seq.causal(kv_heads=1, dim=28, vdim=0, shared=6, size=100)
    assert window.ring == 256 and window.k.shape == (256, 1, 32) and window.v is None and window.shared.shape == (256, 16)
    assert seq.bytes() == 2 * (1024 * 2 * 80 + 256 * 48)


# ── the C ABI ────────────────────────────────────────────────────────────────────────────────

STRUCTS = {"leankv_dense_gemv_t": _native.DenseGemv, "leankv_stream_norm_t": _native.StreamNorm,
           "leankv_causal_attn_t": _native.CausalAttn, "leankv_row_segment_t": _native.RowSegment,
           "leankv_place_rows_t": _native.PlaceRows, "leankv_causal_step_t": _native.CausalStep}


def test_structures_mirror_the_header(tmp_path):
    cc = shutil.which("gcc") or shutil.which("cc")
    if cc is None:
        pytest.skip("no C compiler")
    lines = []
    for c, py in STRUCTS.items():
        lines.append(f'printf("{c} %zu\\n", sizeof({c}));')
        lines += [f'printf("{c}.{f[0]} %zu\\n", offsetof({c}, {f[0]}));' for f in py._fields_]
    (tmp_path / "s.c").write_text('#include <stdio.h>\n#include "leankv_mixers.h"\nint main(void) {' + "\n".join(lines) + "}")
    subprocess.run([cc, "-I", os.path.join(ROOT, "include"), str(tmp_path / "s.c"), "-o", str(tmp_path / "s")], check=True)
    out = dict(l.split() for l in subprocess.run([str(tmp_path / "s")], capture_output=True, text=True).stdout.splitlines())
    for c, py in STRUCTS.items():
        assert int(out[c]) == ctypes.sizeof(py)
        for f in py._fields_:
            assert int(out[f"{c}.{f[0]}"]) == getattr(py, f[0]).offset, f"{c}.{f[0]}"


def test_causal_arguments_are_checked_before_any_launch():
    if torch.cuda.is_available():
        pytest.skip("made-up pointers are only passed where no kernel could be launched")
    lib, fake = _native.mixers(), 0x10000
    make = lambda **kw: _native.CausalAttn(**{**dict(dtype=1, heads=4, kv_heads=2, dim=16, vdim=16, dim_pad=16, vdim_pad=16, size=8,
                                                     scale=1.0, k=fake, v=fake, k_ring=128, k_rows=128), **kw})
    attend = lambda a, rows=1, start=0, ld=64, gate=None: lib.leankv_causal_attend(ctypes.byref(a), fake, gate, 0, fake, ld, rows,
                                                                                 start, None, None)
    assert attend(make(kv_heads=3)) == -1 and attend(make(dim_pad=20)) == -2 and attend(make(dtype=9)) == -5
    assert attend(make(shared_dim=8, shared_pad=16)) == -1                      # no shared part
    assert attend(make(v=None, vdim=32, vdim_pad=32)) == -1                      # values wider than the keys they come from
    assert attend(make(), ld=63) == -1 and attend(make(), gate=fake) == -1
    assert attend(make(), rows=122, start=20) == -6                              # portion + window exceed the ring
    assert attend(make(k_rows=4), rows=5) == -6                                  # rows that are not there
    step = lambda a, **kw: lib.leankv_causal_step(ctypes.byref(a), ctypes.byref(_native.CausalStep(**{**dict(
        q=fake, k_new=fake, v_new=fake, q_stride=16, out=fake, state=fake, max_pos=100), **kw})), None)
    assert step(make(), v_new=None) == -1 and step(make(), rot_own=4) == -1      # rotation without rates
    assert step(make(), rot_own=3, rate=fake) == -1
    assert step(make(size=300), max_pos=300) == -6                               # the ring is shorter than the window
    assert step(make()) == -3                                                    # no workspace
    assert step(make(kv_heads=1), k_gain=fake, rot_own=2, rate=fake) == -1
    place = lambda rows=1, **kw: lib.leankv_place_rows(ctypes.byref(_place(rows, **kw)), None)

    def _place(rows, **kw):
        a = _native.PlaceRows(dtype=1, rows=rows, start=0, n_seg=1)
        a.seg[0] = _native.RowSegment(**{**dict(src=fake, ld=16, heads=1, n=16, dst=fake, dst_ld=16, n_pad=16), **kw})
        return a
    assert place(n_pad=8) == -1 and place(rot=2) == -1 and place(heads=2, gain=fake) == -1 and place(rows=9, ring=8) == -6
    g = _native.DenseGemv(w=fake, x=fake, y=2 * fake, dtype=1, rows=4, cols=8, delta=3 * fake)
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -1                    # a branch without its norm's gain
    g.delta, g.group_rows = None, 3
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -1                    # rows % group_rows
    s = _native.StreamNorm(x_in=fake, x_out=2 * fake, gain=fake, post_gain=fake, dtype=1, delta_dtype=2, rows=1, width=8)
    assert lib.leankv_stream_norm(ctypes.byref(s), None) == -1                   # a post-norm without a branch
