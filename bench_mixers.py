"""``bench.py --workload {rorosun,pefitar}``: the mixer engine beside the framework's closest model at equal size.

For a few layer sizes (random weights): prefill and decode throughput of a Rorosun or Pefitar model and of the
Llama-shaped TEAL + TurboQuant engine with the same width, attention heads and feed-forward (TEAL off: both
stream every weight), then every hot kernel alone with its share of the roofline, next to the like kernel of
the other engine. Launches rotate over the layers, whose weights exceed L2 together.
"""

from __future__ import annotations

import ctypes
import json
import math
import os

ROOT = os.path.dirname(os.path.abspath(__file__))
# name -> width, attention heads / kv heads (x 128), time-mixing heads (x 64), ff, layers
SIZES = {"1k": (1024, 8, 2, 16, 3584, 24), "2k": (2048, 16, 4, 32, 7168, 12), "4k": (4096, 32, 8, 64, 14336, 6)}
VOCAB, WINDOW, POOL, PROMPT = 32768, 1024, 16, 2048
KV_RANK, ROT_DIM, LONG = 512, 64, 32768          # Pefitar's latent layers; positions of the long-context step


def model_config(width, heads, kv, right, ff, layers):
    mixer = {"left": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                      "mask": {"size": WINDOW, "pool": POOL}},
             "right": {"heads": right, "dim": 64}, "left_scale": 0.7, "right_scale": 0.7}
    return {"architecture": "Rorosun", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5},
            "layers": [{"type": "parallel", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}}] * layers}


def pefitar_config(width, heads, kv, _, ff, layers):
    """Attention and latent-attention layers in turn."""
    rot = lambda dims: {"base": 10000.0, "dims": dims}
    mlp = {"kind": "dense", "ff": ff}
    attn = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128,
                                                       "scale": 128 ** -0.5, "rot": rot(128)}}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": 128, "rot_dim": ROT_DIM, "vdim": 128, "q_rank": width // 2, "kv_rank": KV_RANK,
        "mask": {"size": WINDOW}, "scale": (128 + ROT_DIM) ** -0.5, "rot": rot(ROT_DIM)}}
    return {"architecture": "Pefitar", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5},
            "layers": [attn, latent] * (layers // 2), "residual_mult": 0.5, "logit_softcap": 30.0}


def _timed(fn, n_variants, iters, warmup=5):
    import torch

    for i in range(warmup):
        fn(i % n_variants)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(iters):
        fn(i % n_variants)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e-3 / iters


def _graphed(fn, n, reps=20):
    """Seconds per fn(i), the n variants captured in one graph (no host time between launches)."""
    import torch

    s = torch.cuda.Stream()
    with torch.cuda.stream(s):
        for i in range(n):
            fn(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(n):
            fn(i)
    return _timed(lambda _: g.replay(), 1, reps) / n


def _loops(eng, prompt, steps, prefill):
    """(prompt tokens/s, decode tokens/s) on the device."""
    t_pre = _timed(lambda _: prefill(), 1, 5, warmup=3)
    prefill()
    eng.capture()
    t_dec = _timed(lambda _: eng.step(), 1, steps, warmup=8)
    return len(prompt) / t_pre, 1.0 / t_dec


def mixer_leg(size, dev, steps, peaks):
    import torch

    from leankv_b200 import _native
    from leankv_b200.mixer_engine import MixerDecodeEngine, MixerModelConfig
    from leankv_b200.mixers import dtype_code

    width, heads, kv, right, ff, layers = SIZES[size]
    cfg = MixerModelConfig.from_dict(model_config(*SIZES[size]))
    eng = MixerDecodeEngine(cfg, MixerDecodeEngine.random_tensors(cfg, dev), dev, max_seq_len=PROMPT + 2 * steps + 64)
    prompt = torch.randint(0, VOCAB, (PROMPT,), generator=torch.Generator().manual_seed(1)).tolist()

    def prefill():
        eng.reset()
        return eng.extend(prompt, [PROMPT - 1])
    pre, dec = _loops(eng, prompt, steps, prefill)
    lib, L, hbm, tflops = eng.lib, eng.layers, *peaks
    out = {"prefill_tok_s": pre, "decode_tok_s": dec, "launches_per_step": eng.launches_per_step,
           "state_bytes": eng.seq.bytes(), "kernels": {}}
    st = lambda: torch.cuda.current_stream().cuda_stream

    def mem(name, seconds, nbytes):
        out["kernels"][name] = {"us": seconds * 1e6, "gbs": nbytes / seconds / 1e9, "frac": nbytes / seconds / 1e9 / hbm,
                                "bound": "hbm"}

    def math_(name, seconds, flops):
        out["kernels"][name] = {"us": seconds * 1e6, "tflops": flops / seconds / 1e12,
                                "frac": flops / seconds / 1e12 / tflops, "bound": "tensor"}

    gemv = lambda a: _native.check(lib.leankv_dense_gemv(ctypes.byref(a), st()), "gemv", lib)
    mem("gemv_in_norm_shift", _graphed(lambda i: gemv(L[i].mixer._step_args[0]), layers), 2 * L[0].mixer.w_in.numel())
    mem("gemv_out_residual", _graphed(lambda i: gemv(L[i].mixer._step_args[2]), layers), 2 * L[0].mixer.w_out.numel())
    mem("gemv_gate_up_silu", _graphed(lambda i: gemv(L[i].mlp._step_args[0]), layers), 2 * L[0].mlp.w_gu.numel())
    mem("gemv_down_residual", _graphed(lambda i: gemv(L[i].mlp._step_args[1]), layers), 2 * L[0].mlp.w_down.numel())
    mem("gemv_head", _graphed(lambda i: gemv(eng._head_args), 4), 2 * eng.head.numel())
    n_keys = WINDOW + (eng.pos - WINDOW + 1) // POOL
    m0 = L[0].mixer

    def mixers(i, l=True, r=True):
        m = L[i].mixer
        _native.check(lib.leankv_mixer_step(ctypes.byref(m.left.c) if l else None, ctypes.byref(m.right.c) if r else None,
                                            ctypes.byref(m._step_args[1]), st()), "mixer_step", lib)
    kv_bytes, s_bytes = n_keys * kv * 256 * 2, 2 * right * 64 * 64 * 4
    eng.state[0] = eng.pos
    mem("mixer_step", _graphed(mixers, layers), kv_bytes + s_bytes)
    mem("mixer_step_left_only", _graphed(lambda i: mixers(i, r=False), layers), kv_bytes)
    mem("mixer_step_right_only", _graphed(lambda i: mixers(i, l=False), layers), s_bytes)

    # prompt kernels on a portion of PROMPT tokens
    T, W = PROMPT, width
    x, d = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
    h = torch.empty(T, W, dtype=eng.dtype, device=dev)
    mixed = torch.empty(5, T, W, dtype=eng.dtype, device=dev)
    mem("stream_norm_shift", _graphed(lambda i: eng._stream_norm(x, L[i].first.norm, h, d, L[i].first, L[i].mixer, mixed), layers),
        T * W * (4 * 3 + 2 * 6))
    mem("stream_norm", _graphed(lambda i: eng._stream_norm(x, L[i].second.norm, h, d, L[i].second), layers), T * W * (4 * 3 + 2))
    gu = torch.randn(T, 2 * ff, device=dev).bfloat16()
    act = torch.empty(T, ff, dtype=eng.dtype, device=dev)
    mem("silu_mul", _graphed(lambda i: lib.leankv_silu_mul(gu.data_ptr(), act.data_ptr(), 1, T, ff, st()), 4), T * ff * 6)
    qkv = torch.randn(T, m0.left.spec.qkv_width, device=dev)
    q = torch.empty(T, heads, 128, dtype=eng.dtype, device=dev)
    cat = torch.empty(T, m0.out_width, dtype=eng.dtype, device=dev)
    mem("window_pool_append", _graphed(lambda i: lib.leankv_window_pool_append(
        ctypes.byref(L[i].mixer.left.c), qkv.data_ptr(), qkv.stride(0), L[i].mixer.bias.data_ptr(), q.data_ptr(), T, 0,
        st()), layers), T * qkv.shape[1] * 6)
    need = lib.leankv_window_pool_workspace_bytes(ctypes.byref(m0.left.c), T, T)
    ws = torch.empty(max(need, 16), dtype=torch.uint8, device=dev)
    pairs = sum(min(i + 1, WINDOW) + max(0, i - WINDOW + 1) // POOL for i in range(T))
    math_("window_pool_attend", _graphed(lambda i: lib.leankv_window_pool_attend(
        ctypes.byref(L[i].mixer.left.c), q.data_ptr(), cat.data_ptr(), cat.stride(0), 0.7, T, 0, ws.data_ptr(),
        ws.numel(), st()), layers), 2 * pairs * heads * (128 + 128 + heads))
    N = right * 64
    rkvg = torch.randn(4, T, N, device=dev).bfloat16()
    z = torch.randn(T, N, device=dev)
    need = lib.leankv_time_mix_workspace_bytes(ctypes.byref(m0.right.c), T)
    ws2 = torch.empty(need, dtype=torch.uint8, device=dev)
    t = _graphed(lambda i: lib.leankv_time_mix_rows(
        ctypes.byref(L[i].mixer.right.c), *(rkvg[j].data_ptr() for j in range(4)), z.data_ptr(), cat.data_ptr(),
        cat.stride(0), 0.7, T, ws2.data_ptr(), ws2.numel(), st()), layers)
    mem("time_mix_rows", t, T * N * (4 * 2 + 4 + 2))
    out["kernels"]["time_mix_rows"]["fp32_tflops"] = T * N * 64 * 6 / t / 1e12
    return out


def pefitar_leg(size, dev, steps, peaks):
    import torch

    from leankv_b200 import _native
    from leankv_b200.mixer_engine import MixerDecodeEngine, MixerModelConfig

    width, heads, kv, _, ff, layers = SIZES[size]
    cfg = MixerModelConfig.from_dict(pefitar_config(*SIZES[size]))
    eng = MixerDecodeEngine(cfg, MixerDecodeEngine.random_tensors(cfg, dev), dev, max_seq_len=LONG, max_chunk=PROMPT)
    prompt = torch.randint(0, VOCAB, (PROMPT,), generator=torch.Generator().manual_seed(1)).tolist()

    def prefill():
        eng.reset()
        return eng.extend(prompt, [PROMPT - 1])
    pre, dec = _loops(eng, prompt, steps, prefill)
    lib, hbm, tflops = eng.lib, *peaks
    out = {"prefill_tok_s": pre, "decode_tok_s": dec, "launches_per_step": eng.launches_per_step,
           "state_bytes": eng.seq.bytes(), "kernels": {}}
    st = lambda: torch.cuda.current_stream().cuda_stream
    runs, attn, latent = eng.layers, eng.layers[0::2], eng.layers[1::2]
    n = len(attn)

    def mem(name, seconds, nbytes):
        out["kernels"][name] = {"us": seconds * 1e6, "gbs": nbytes / seconds / 1e9, "frac": nbytes / seconds / 1e9 / hbm,
                                "bound": "hbm"}

    def math_(name, seconds, flops):
        out["kernels"][name] = {"us": seconds * 1e6, "tflops": flops / seconds / 1e12,
                                "frac": flops / seconds / 1e12 / tflops, "bound": "tensor"}

    gemv = lambda a: _native.check(lib.leankv_dense_gemv(ctypes.byref(a), st()), "gemv", lib)
    A, L = attn[0].mixer, latent[0].mixer
    mem("gemv_qkvg_join_norm", _graphed(lambda i: gemv(attn[i].mixer._step_args[0]), n), 2 * A.w_in.numel())
    mem("gemv_out", _graphed(lambda i: gemv(attn[i].mixer._step_args[2]), n), 2 * A.w_out.numel())
    for k, name, w in ((0, "gemv_latent_in", L.w_down), (1, "gemv_latent_q", L.w_q), (2, "gemv_latent_fold", L.w_fold),
                       (4, "gemv_latent_unfold", L.w_unfold), (5, "gemv_latent_out", L.w_out)):
        mem(name, _graphed(lambda i: gemv(latent[i].mixer._step_args[k]), n), 2 * w.numel())
    mem("gemv_gate_up_silu", _graphed(lambda i: gemv(runs[i].mlp._step_args[0]), layers), 2 * runs[0].mlp.w_gu.numel())
    mem("gemv_down", _graphed(lambda i: gemv(runs[i].mlp._step_args[1]), layers), 2 * runs[0].mlp.w_down.numel())
    mem("gemv_head", _graphed(lambda i: gemv(eng._head_args), 4), 2 * eng.head.numel())

    def step(r, k):
        m = r.mixer
        _native.check(lib.leankv_causal_step(ctypes.byref(m.c), ctypes.byref(m._step_args[k]), st()), "causal_step", lib)
    for name, pos in (("causal_step", eng.pos), ("causal_step_32k", LONG - 1)):
        eng.state[0] = pos
        mem(name, _graphed(lambda i: step(attn[i], 1), n), 2 * pos * kv * 256)
    mem("causal_step_latent", _graphed(lambda i: step(latent[i], 3), n), 2 * WINDOW * (KV_RANK + ROT_DIM))

    # prompt kernels on a portion of PROMPT tokens
    T, W = PROMPT, width
    x, d = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
    h = torch.empty(T, W, dtype=eng.dtype, device=dev)
    mem("stream_norm_join", _graphed(lambda i: eng._stream_norm(x, runs[i].second.norm, h, d, runs[i].second), layers),
        T * W * (4 * 3 + 2))
    gu = torch.randn(T, 2 * ff, device=dev).bfloat16()
    act = torch.empty(T, ff, dtype=eng.dtype, device=dev)
    mem("silu_mul", _graphed(lambda i: lib.leankv_silu_mul(gu.data_ptr(), act.data_ptr(), 1, T, ff, st()), 4), T * ff * 6)
    y = torch.randn(T, A.in_width, device=dev)
    mem("place_rows", _graphed(lambda i: attn[i].mixer.place(y, 0), n), T * A.at_g * 6)
    q = attn[0].mixer.place(y, 0)
    gate = y[:, A.at_g:]
    math_("causal_attend", _graphed(lambda i: attn[i].mixer._attend(attn[i].mixer.c, q, gate, 0), n),
          2 * T * (T + 1) // 2 * heads * 256)
    z = torch.randn(T, heads * (128 + ROT_DIM), device=dev)
    ql = L.place_q(z, 0)
    mem("place_rows_latent_q", _graphed(lambda i: latent[i].mixer.place_q(z, 0), n), T * z.shape[1] * 6)
    math_("latent_expand", _graphed(lambda i: latent[i].mixer._expanded(0, T), n), 2 * T * KV_RANK * heads * 256)
    e, keep = L._expanded(0, T)
    pairs = sum(min(i + 1, WINDOW) for i in range(T))
    math_("causal_attend_latent", _graphed(lambda i: L._attend(e, ql, None, 0), n), 2 * pairs * heads * (256 + ROT_DIM))
    del keep
    return out


def llama_leg(size, dev, steps, peaks):
    """The Llama-shaped engine (3-bit KV pages, TEAL off) at the same width, heads, ff and layers."""
    import torch

    from leankv_b200 import _native
    from leankv_b200.engine import DecodeEngine, DecoderConfig

    width, heads, kv, _, ff, layers = SIZES[size]
    cfg = DecoderConfig(vocab_size=VOCAB, hidden_size=width, intermediate_size=ff, num_layers=layers,
                        num_q_heads=heads, num_kv_heads=kv)
    eng = DecodeEngine.random_init(cfg, dev, max_seq_len=PROMPT + 2 * steps + 64)
    prompt = torch.randint(0, VOCAB, (PROMPT,), generator=torch.Generator().manual_seed(1)).tolist()
    pre, dec = _loops(eng, prompt, steps, lambda: eng.prefill(prompt))
    lib, hbm, tflops = eng.lib, *peaks
    out = {"prefill_tok_s": pre, "decode_tok_s": dec, "launches_per_step": eng.launches_per_step, "kernels": {}}
    W = eng.w["layers"]
    st = eng._st

    def mem(name, seconds, nbytes):
        out["kernels"][name] = {"us": seconds * 1e6, "gbs": nbytes / seconds / 1e9, "frac": nbytes / seconds / 1e9 / hbm,
                                "bound": "hbm"}
    mem("gemv_qkv_norm", _graphed(lambda i: eng._gemv(W[i]["wqkv_t"], eng.h, eng.qkv, 0.0, eng._qkv_segments(i),
                                                      norm_w=W[i]["ln1"]), layers), 2 * W[0]["wqkv_t"].numel())
    mem("gemv_o_residual", _graphed(lambda i: eng._gemv(W[i]["wo_t"], eng.attn, eng.h, -1.0, residual=eng.h), layers),
        2 * W[0]["wo_t"].numel())
    mem("gemv_gate_up_silu", _graphed(lambda i: lib.leankv_sparse_swiglu_rmsnorm_f16(
        W[i]["wgate_t"].data_ptr(), W[i]["wup_t"].data_ptr(), eng.h.data_ptr(), W[i]["ln2"].data_ptr(), cfg.rms_eps,
        eng.mlp_h.data_ptr(), eng.inter, width, -1.0, -1.0, eng.ws_gemv.data_ptr(), eng.ws_gemv.numel(),
        eng.active_elems.data_ptr(), st()), layers), 4 * W[0]["wgate_t"].numel())
    mem("gemv_down_residual", _graphed(lambda i: eng._gemv(W[i]["wdown_t"], eng.mlp_h, eng.h, -1.0, residual=eng.h),
                                       layers), 2 * W[0]["wdown_t"].numel())
    mem("gemv_head", _graphed(lambda i: eng._gemv(eng.w["lm_head_t"], eng.h, eng.logits, -1.0,
                                                  norm_w=eng.w["final_norm"]), 4), 2 * eng.w["lm_head_t"].numel())
    sp, n_tok = eng.state.data_ptr(), int(eng.state[0])

    def attn(i):
        _native.check(lib.leankv_tq_decode_attn_rotated(
            eng.q_rot.data_ptr(), eng.attn.data_ptr(), 1, eng.nq, eng.nkv, eng.pools[i].data_ptr(), eng.max_pages, sp + 8,
            eng.page_indices.data_ptr(), sp + 16, eng.max_pages, eng.Pi_v[i].data_ptr(), eng.centroids_host.data_ptr(),
            1.0 / math.sqrt(128.0), eng.ws_attn.data_ptr(), eng.ws_attn.numel(), 0, st()), "attn")
    mem("decode_attn", _graphed(attn, layers), 2 * kv * n_tok * 50)
    T = PROMPT
    q, o = torch.randn(T, heads, 128, device=dev).half(), torch.empty(T, heads, 128, device=dev).half()
    need = lib.leankv_tq_prefill_attn_workspace_bytes(T, 0, eng.nq, eng.nkv)
    ws = torch.zeros(need, dtype=torch.uint8, device=dev)
    t = _graphed(lambda i: lib.leankv_tq_prefill_attn(
        q.data_ptr(), o.data_ptr(), T, 0, eng.nq, eng.nkv, eng.pools[i].data_ptr(), eng.max_pages,
        eng.page_indices.data_ptr(), eng.Pi_k[i].data_ptr(), eng.Pi_v[i].data_ptr(), eng.centroids_host.data_ptr(),
        1.0 / math.sqrt(128.0), ws.data_ptr(), ws.numel(), st()), layers)
    flops = 4 * T * (T + 1) // 2 * heads * 128
    out["kernels"]["prefill_attn"] = {"us": t * 1e6, "tflops": flops / t / 1e12, "frac": flops / t / 1e12 / tflops,
                                      "bound": "tensor"}
    x = torch.randn(T, width, device=dev).half()
    y, d = torch.empty_like(x), torch.randn(T, width, device=dev).half()
    mem("rmsnorm_rows", _graphed(lambda i: lib.leankv_rmsnorm_rows_f16(
        x.data_ptr(), d.data_ptr(), W[i]["ln1"].data_ptr(), y.data_ptr(), T, width, 1e-5, st()), layers),
        T * width * 2 * 4)
    gu, act = torch.randn(T, 2 * ff, device=dev).half(), torch.empty(T, ff, device=dev).half()
    mem("silu_mul", _graphed(lambda i: lib.leankv_silu_mul_f16(gu.data_ptr(), act.data_ptr(), T, ff, st()), 4), T * ff * 6)
    return out


def run(args, sampler_cls):
    import torch

    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        peaks, source = (float(p["hbm_gbs"]), float(p["bf16_tflops"])), "measured"
    except OSError:
        peaks, source = (6650.0, 1590.0), "fallback"
    steps = args.steps if args.steps_given else 128
    sizes = [s for s in args.sizes.split(",") if s]
    sampler = sampler_cls(0)
    sampler.start()
    result, name = {}, args.workload
    legs = {"rorosun": mixer_leg, "pefitar": pefitar_leg}
    for s in sizes:
        result[s] = {name: legs[name](s, dev, steps, peaks)}
        torch.cuda.empty_cache()
        result[s]["llama_same_size"] = llama_leg(s, dev, steps, peaks)
        torch.cuda.empty_cache()
    sampler.stop()
    last = result[sizes[-1]][name]
    more = {"pool": POOL} if name == "rorosun" else {"kv_rank": KV_RANK, "rot_dim": ROT_DIM, "long_context": LONG}
    columns = ("width", "heads", "kv_heads", "time_mix_heads" if name == "rorosun" else None, "ff", "layers")
    print(json.dumps({
        "metric": f"B=1 decode tok/s ({name.capitalize()} layers, largest size)", "value": last["decode_tok_s"],
        "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 8, "higher_is_better": True, "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic", "clocks": sampler.summary(),
        "peaks": {"hbm_gbs": peaks[0], "bf16_tflops": peaks[1], "source": source},
        "config": {"sizes": {s: {c: v for c, v in zip(columns, SIZES[s]) if c} for s in sizes},
                   "vocab": VOCAB, "window": WINDOW, "prompt_len": PROMPT, **more,
                   "l2": "launches rotate over the layers; their weights exceed L2 together"},
        "sizes": result}))
