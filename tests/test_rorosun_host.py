"""Rorosun without a GPU: the plain implementation's own properties, configuration and checkpoint reading,
the registry, the sequence state, the replay loop and the C ABI of the mixer library."""

import copy
import ctypes
import io
import json
import math
import os
import re
import subprocess
import sys

import pytest
import torch

from conftest import ROOT
from leankv_b200 import _native, checkpoint, registry, trace
from leankv_b200.mixer_engine import MixerModelConfig
from leankv_b200.mixers import TimeMixSpec, WindowPoolSpec
from leankv_b200.sequence_state import SequenceState
from oracle import rorosun as plain
from rorosun_util import config, layer, tokens, weights, write_model, write_safetensors


# ── the plain implementation ─────────────────────────────────────────────────────────────────

def test_visibility_by_enumeration():
    for size, pool in ((1, 1), (5, 3), (4, 4), (3, 7), (8, 2)):
        tok, blk = plain.visible(40, size, pool)
        for i in range(40):
            assert tok[i].nonzero().flatten().tolist() == [j for j in range(40) if 0 <= i - j < size]
            seen = [b for b in range(40 // pool) if all(i - j >= size for j in range(b * pool, (b + 1) * pool))]
            assert blk[i].nonzero().flatten().tolist() == seen


def test_recurrence_against_the_unrolled_sum():
    T, H, d = 7, 2, 3
    g = torch.Generator().manual_seed(0)
    r, k, v = (torch.randn(T, H, d, generator=g, dtype=torch.float64) for _ in range(3))
    w = torch.rand(T, H, d, generator=g, dtype=torch.float64)
    u = torch.randn(H, d, generator=g, dtype=torch.float64)
    o, S = plain.wkv(r, k, v, w, u)
    for t in range(T):
        want = torch.zeros(H, d, dtype=torch.float64)
        for j in range(t + 1):
            a = u if j == t else w[j + 1:t].prod(0)      # decays of the tokens strictly between
            want += (r[t] * a * k[j]).sum(-1, keepdim=True) * v[j]
        assert torch.allclose(o[t], want)
    o2, S2 = plain.wkv(r[:4], k[:4], v[:4], w[:4], u)
    o3, S3 = plain.wkv(r[4:], k[4:], v[4:], w[4:], u, S2)
    assert torch.allclose(torch.cat([o2, o3]), o) and torch.allclose(S3, S)


def test_plain_model_is_causal_and_every_parameter_matters():
    cfg = config()
    w, ids = weights(cfg), tokens(cfg, 24)
    full = plain.forward(cfg, w, ids)
    assert torch.allclose(plain.forward(cfg, w, ids[:17]), full[:17])
    for name in w:
        ch = {n: t.float() * (1.25 if n == name else 1.0) + (0.1 if n == name else 0.0) for n, t in w.items()}
        assert not torch.allclose(plain.forward(cfg, ch, ids), full, atol=1e-6), f"{name} has no effect"


@pytest.mark.parametrize("key", ["size", "pool", "scale", "left_scale", "right_scale"])
def test_plain_model_reads_every_constant(key):
    cfg = config()
    w, ids = weights(cfg), tokens(cfg, 24)
    other = copy.deepcopy(cfg)
    m = other["layers"][0]["mixer"]
    if key in ("size", "pool"):
        m["left"]["mask"][key] += 1
    elif key == "scale":
        m["left"]["scale"] *= 1.5
    else:
        m[key] *= 1.5
    assert not torch.allclose(plain.forward(other, w, ids), plain.forward(cfg, w, ids), atol=1e-6)


# ── configuration, checkpoints, registry ─────────────────────────────────────────────────────

def test_config_reading():
    c = config(vocab=31, width=24, eps=3e-4)
    m = MixerModelConfig.from_dict(json.loads(json.dumps(c)))
    assert (m.vocab_size, m.hidden_size, m.eps, len(m.layers)) == (31, 24, 3e-4, 3)
    s = WindowPoolSpec.from_dict(c["layers"][0]["mixer"]["left"])
    assert s == WindowPoolSpec(4, 2, 16, 24, 10, 3, 0.3)
    assert (s.q_width, s.qkv_width, s.out_width) == (64, 64 + 32 + 48, 96)
    for change in (lambda d: d.update(extra=1), lambda d: d["norm"].update(offset=1),
                   lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0].update(gate=1)):
        bad = copy.deepcopy(c)
        change(bad)
        with pytest.raises(ValueError):
            MixerModelConfig.from_dict(bad)
    left = copy.deepcopy(c["layers"][0]["mixer"]["left"])
    left["kv_heads"] = 3
    with pytest.raises(ValueError):
        WindowPoolSpec.from_dict(left)
    left["kv_heads"], left["mask"]["sinks"] = 2, 4
    with pytest.raises(ValueError):
        WindowPoolSpec.from_dict(left)
    with pytest.raises(ValueError):
        TimeMixSpec.from_dict({"heads": 0, "dim": 4})


def test_safetensors_round_trip(tmp_path):
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.randn(()).bfloat16(), "c": torch.randn(7)}
    write_safetensors(tmp_path / "model.safetensors", t)
    got = checkpoint.read_weights(str(tmp_path))
    assert set(got) == set(t)
    for n in t:
        assert got[n].dtype == t[n].dtype and got[n].shape == t[n].shape and torch.equal(got[n], t[n])
    write_safetensors(tmp_path / "x-1.safetensors", {"a": t["a"]})
    write_safetensors(tmp_path / "x-2.safetensors", {"c": t["c"]})
    os.unlink(tmp_path / "model.safetensors")
    (tmp_path / "model.safetensors.index.json").write_text(json.dumps(
        {"weight_map": {"a": "x-1.safetensors", "c": "x-2.safetensors"}}))
    assert set(checkpoint.read_weights(str(tmp_path))) == {"a", "c"}


def test_tensor_bag_refuses_what_does_not_fit():
    bag = checkpoint.TensorBag({"a": torch.zeros(2, 3), "b": torch.zeros(4)})
    assert bag.take("a", 2, 3).shape == (2, 3)
    with pytest.raises(ValueError, match="shape"):
        bag.take("b", 5)
    with pytest.raises(ValueError, match="no tensor"):
        bag.take("c", 5)
    with pytest.warns(UserWarning, match="no layer uses"):
        bag.finish()


def test_registry_knows_the_models(tmp_path):
    assert {"Rorosun", "LlamaForCausalLM", "MistralForCausalLM"} <= set(registry.architectures())
    assert registry.supports({"architecture": "Rorosun"}, "float32")
    assert not registry.supports({"architectures": ["LlamaForCausalLM"]}, "float32")
    with pytest.raises(ValueError, match="not one of"):
        registry.architecture_of({"architecture": "Unknown"})
    folder = write_model(tmp_path / "m", config(), weights(config()))
    with pytest.raises(ValueError, match="float16"):
        registry.load_engine(folder, dtype="float16")
    if not torch.cuda.is_available():
        with pytest.raises(RuntimeError, match="GPU"):
            registry.load_engine(folder)


def test_command_line_lists_architectures_and_refuses_a_type():
    out = subprocess.run([sys.executable, "-m", "leankv_b200", "architectures"], cwd=ROOT, capture_output=True, text=True)
    assert out.returncode == 0 and "Rorosun" in out.stdout.split()


def test_trace_run_refuses_a_type_the_model_lacks(tmp_path):
    folder = tmp_path / "m"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps({"architectures": ["LlamaForCausalLM"]}))
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32",
                          "--out", str(tmp_path), "--max-tokens", "8"], capture_output=True, text=True)
    assert out.returncode == trace.REFUSED


class _FakeEngine:
    """Logits row = (tokens so far in this sequence, token)."""

    def __init__(self):
        self.n, self.resets = 0, 0

    def reset(self):
        self.n = 0
        self.resets += 1

    def extend(self, toks, want):
        rows = [[self.n + w, toks[w]] for w in want]
        self.n += len(toks)
        return torch.tensor(rows, dtype=torch.float32).reshape(len(want), 2)


def test_replay_loop(tmp_path):
    eng, said = _FakeEngine(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    trace.replay(eng, (json.dumps(s) + "\n" for s in steps), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"]
    got = torch.frombuffer(bytearray((tmp_path / "0.f32").read_bytes()), dtype=torch.float32)
    assert got.tolist() == [2, 7, 0, 5]
    assert not (tmp_path / "1.f32").exists()
    assert torch.frombuffer(bytearray((tmp_path / "2.f32").read_bytes()), dtype=torch.float32).tolist() == [0, 9]
    bad = [{"step": 0, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": []},
           {"step": 1, "entries": [{"id": "b", "tokens": [1], "want": []}], "end": []}]
    with pytest.raises(ValueError, match="before a has ended"):
        trace.replay(_FakeEngine(), map(json.dumps, bad), str(tmp_path), said.append)


def test_windows_longer_than_the_sequence_take_no_more_memory():
    spec = WindowPoolSpec(4, 2, 16, 24, size=1 << 20, pool=1 << 16, scale=1.0)
    assert spec.bounded(100) == WindowPoolSpec(4, 2, 16, 24, size=100, pool=101, scale=1.0)
    assert spec.bounded(1 << 21) == spec
    for n in (1, 2, 50, 100):            # no position below the bound sees anything else
        a, b = plain.visible(n, spec.size, spec.pool), plain.visible(n, 100, 101)
        assert torch.equal(a[0], b[0]) and a[1].shape[1] == b[1].shape[1] == 0


def test_sequence_state_sizes_and_reset():
    seq = SequenceState("cpu", torch.bfloat16, max_seq_len=100, max_chunk=16)
    w = seq.window(kv_heads=2, dim=10, vdim=24, size=7, pool=12)
    assert w.k_ring.shape == (12 + 15, 2, 16) and w.v_ring.shape == (27, 2, 32)
    assert w.k_pool.shape == (8, 2, 16) and w.ring == 27 and w.max_blocks == 8
    c = seq.carried(3, 4, 4)
    c.fill_(2.0)
    seq.reset()
    assert float(c.abs().max()) == 0.0 and seq.carried_tensors[0] is c
    assert seq.bytes() == 2 * (27 * 2 * 48 + 8 * 2 * 48) + 4 * 48


# ── the C ABI ────────────────────────────────────────────────────────────────────────────────

def test_mixer_library_exports_every_declared_symbol():
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "leankv_mixers.h")).read(), flags=re.S)
    names = sorted(set(re.findall(r"\b(leankv_[a-z0-9_]+)\s*\(", text)))
    assert names == sorted(_native.MIXER_SIGNATURES)
    lib = _native.mixers()
    for n in names:
        assert hasattr(lib, n)


def test_mixer_arguments_are_checked_before_any_launch():
    if torch.cuda.is_available():
        pytest.skip("made-up pointers are only passed where no kernel could be launched")
    lib, fake = _native.mixers(), 0x10000
    g = _native.DenseGemv(w=fake, x=fake, y=fake, dtype=1, rows=4, cols=8)
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -1                 # y aliases x
    g.y, g.dtype = fake * 2, 7
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -5
    g.dtype, g.residual = 1, fake
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -1                 # residual without scale
    g.residual, g.n_mix = None, 1
    assert lib.leankv_dense_gemv(ctypes.byref(g), None) == -1                 # shift without prev
    w = _native.WindowPool(dtype=1, heads=4, kv_heads=3, dim=16, vdim=16, dim_pad=16, vdim_pad=16, size=4, pool=2,
                           ring=8, max_blocks=4, scale=1.0, k_ring=fake, v_ring=fake, k_pool=fake, v_pool=fake)
    call = lambda rows, start=0: lib.leankv_window_pool_append(ctypes.byref(w), fake, 256, None, fake, rows, start, None)
    assert call(1) == -1                                                      # heads % kv_heads
    w.kv_heads, w.dim_pad = 2, 20
    assert call(1) == -2
    w.dim_pad = 16
    assert call(6) == -6                                                      # portion + window exceed the ring
    attend = lambda rows, start: lib.leankv_window_pool_attend(ctypes.byref(w), fake, fake, 64, 1.0, rows, start, None,
                                                               0, None)
    assert attend(2, 20) == -6                                                # more blocks than there are
    t = _native.TimeMix(dtype=1, heads=2, dim=8, S=fake, u=fake, w0=fake, norm=fake, eps=1e-5)
    args = [fake] * 6
    assert lib.leankv_time_mix_rows(ctypes.byref(t), *args, 16, 1.0, 4, None, 0, None) == -3
    assert lib.leankv_time_mix_rows(ctypes.byref(t), *args, 8, 1.0, 4, None, 0, None) == -1
    s = _native.StreamNorm(x_in=fake, x_out=fake, delta=fake, scale=fake, gain=fake, dtype=1, delta_dtype=2, rows=1,
                           width=8)
    assert lib.leankv_stream_norm(ctypes.byref(s), None) == -1                # in place
