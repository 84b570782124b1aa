"""Throughput of the hybrid family beside the closest transformer of the same size (``bench.py --family hybrid``).

For each width a 4-layer hybrid model (latent attention, gated delta rule, gated linear attention, latent attention;
dense erf-GELU feed-forward of 4x width) and a 4-layer Llama-style transformer of the same width (GQA, gated MLP
sized to the same parameter count) are built with random weights.  Measured with CUDA events after warm-up:

* prefill: one prompt of ``prompt_len`` tokens, tokens/s;
* decode: one token per step at a context of ``prompt_len`` tokens, tokens/s, for one stream (what the transformer
  engine's recurrent pipeline runs per stage) and for a batch of streams (hybrid only: its runner batches);
* the hybrid family's own kernels one by one on the prefill shapes and on the decode shapes, with achieved bytes/s
  and FLOP/s against the measured peaks, beside the transformer's attention kernels on the same token counts.

An L2 flush (a write larger than L2) separates timed iterations of the single-kernel measurements.

``bench.py --family vudelix`` measures the pre-norm design of the family (windowed grouped-query attention, gated
delta rule, mixture-of-experts and dense feed-forwards, per-layer token embedding) the same way, beside the sandwich
design of the same width as the closest existing model, with its own kernels one by one.

``bench.py --family labepel`` measures the parallel-block design (chunk-masked attention with a softmax sink and value
mixing, softmax-routed gated experts plus a shared expert, layer scale, learned positions) beside the pre-norm design
of the same width, whose windowed attention and mixture of experts are the closest existing kernels.  Decoding is
timed inside one chunk (the prompt ends short of a chunk edge), so that a step sees about as many keys as the
windowed design does.

``bench.py --family ratesun`` measures the sandwich design with input convolutions, an average over depth, windowed
latent attention on shared caches and a polynomial activation beside the plain sandwich design of the same width.

``bench.py --family zudovik`` measures the post-norm design (causal grouped-query attention with the norm over the
whole q and k projections, a score cap and learned sinks, a layer on another layer's keys and values, the fixed-decay
linear recurrence, clamped gated experts with identity experts and a token-gated shared expert) beside the
parallel-block design of the same width, whose attention and mixture of experts are the closest existing kernels; the
recurrence is set beside the gated linear attention of the sandwich design, timed in the same run.

``bench.py --family dufelix`` measures the RMS sandwich design (grouped-query attention, latent attention with sinks, state-space
recurrence, gated feed-forward) beside the depth-averaged design of the same width, its closest model as a whole; single
kernels also stand beside the post-norm design's grouped-query attention and recurrence and the sandwich design's convolution.
"""
from __future__ import annotations

import json
import os
from typing import Any, Callable, Dict, List

import torch

__all__ = ["run_family_compare", "hybrid_bench_config", "vudelix_bench_config", "labepel_bench_config", "zudovik_bench_config",
           "ratesun_bench_config", "dufelix_bench_config"]


def dufelix_bench_config(width: int) -> Dict[str, Any]:
    """4 layers: attention, latent attention, two recurrences (the second with the first one's sizes and its own weights), each
    with a gated feed-forward whose three matrices have as many weights as a dense ``4 * width`` one.  Attention sizes are
    those of the other designs' bench models; the recurrence is twice as wide as the stream, heads of 64, state 128."""
    h = width // 128
    yarn = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    att = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
           "rot": {"dims": 64, "base": 500000.0, "scaling": yarn}}
    lat = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": min(1536, width), "scale": 192 ** -0.5,
           "rot": {"dims": 64, "base": 10000.0, "scaling": yarn}}
    ssm = {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8}
    mlp = {"kind": "dense", "ff": (8 * width // 3 + 63) // 64 * 64}
    layers = [{"type": t, "mixer": dict(m), "mlp": dict(mlp)}
              for t, m in (("attention", att), ("latent_attention", lat), ("mamba2", ssm), ("mamba2", ssm))]
    return {"architecture": "Dufelix", "vocab": 32000, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "embedding": {"scale": 32.0}}


def ratesun_bench_config(width: int, window: int = 1024) -> Dict[str, Any]:
    """4 layers of windowed latent attention + dense (polynomial activation, ``4 * width``), the second and the fourth on the
    cache of the layer before; attention sizes of the sandwich design's bench model."""
    h = width // 128
    lat = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": min(1536, width),
           "scale": 192 ** -0.5, "rot": {"dims": 64, "base": 10000.0}, "mask": {"size": window}}
    mlp = {"kind": "dense", "ff": 4 * width}
    layers = [{"type": "latent_attention", "mixer": dict(lat) if i % 2 == 0 else dict(lat, kv_from=i - 1), "mlp": dict(mlp)}
              for i in range(4)]
    return {"architecture": "Ratesun", "vocab": 32000, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 50021, "mul_prev": 1009, "mul_cur": 31}}, "canon": {"taps": 4},
            "residual_mult": 0.5, "token_side": {"dim": 64}, "logit_scale": 0.5}


def zudovik_bench_config(width: int) -> Dict[str, Any]:
    """4 layers: attention + dense (squared ReLU, ``4 * width``), recurrence + experts, attention + experts, attention on
    the third layer's keys and values + experts.  Two of eight clamped experts of width ``width`` plus two identity
    outputs in the router, and a token-gated shared expert of width ``width`` (the parallel-block design's expert sizes)."""
    h = width // 128
    att = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0,
           "rot": {"dims": 64, "base": 500000.0}}
    lit = {"heads": h, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-3 - 5 * i / max(1, h - 1)) for i in range(h)]}
    moe = {"kind": "moe", "expert": {"ff": width, "limit": 7.0}, "router": {"experts": 8, "identity": 2, "top": 2},
           "shared": {"ff": width, "limit": 7.0}}
    layers = [{"type": "attention", "mixer": dict(att), "mlp": {"kind": "dense", "ff": 4 * width}},
              {"type": "lightning", "mixer": lit, "mlp": dict(moe)}, {"type": "attention", "mixer": dict(att), "mlp": dict(moe)},
              {"type": "attention", "mixer": {**att, "kv_from": 2}, "mlp": dict(moe)}]
    return {"architecture": "Zudovik", "vocab": 32000, "width": width, "embedding": {"scale": 32.0}, "layers": layers,
            "norm": {"eps": 1e-6}}


def vudelix_bench_config(width: int, window: int = 1024) -> Dict[str, Any]:
    """4 layers: delta + dense, attention + experts, delta + experts, attention + dense.  Two of eight experts of
    width ``2 * width`` per token, so a token's feed-forward work equals the dense ``4 * width`` one."""
    h = width // 128
    dense = {"kind": "dense", "ff": 4 * width}
    moe = {"kind": "moe", "expert": {"ff": 2 * width}, "router": {"experts": 8, "top": 2}}
    att = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": window},
           "rot": {"dims": 128, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    delta = {"heads": h, "kv_heads": max(1, h // 2), "dim": 128, "vdim": 128, "conv": 4}
    layers = [{"type": "channel_delta", "mixer": dict(delta), "mlp": dense}, {"type": "attention", "mixer": dict(att), "mlp": moe},
              {"type": "channel_delta", "mixer": dict(delta), "mlp": moe}, {"type": "attention", "mixer": dict(att), "mlp": dense}]
    return {"architecture": "Vudelix", "vocab": 32000, "width": width, "layers": layers, "norm": {"eps": 1e-6},
            "residual_mult": 0.5, "token_side": {"dim": 64}}


def labepel_bench_config(width: int, chunk: int = 1024, positions: int = 8192) -> Dict[str, Any]:
    """4 attention layers with experts: two of eight gated experts of width ``width`` per token plus a shared expert of
    the same width (9 width^2 weights per token, the dense ``4 * width`` feed-forward has 8)."""
    h = width // 128
    att = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": chunk},
           "v_mix": True}
    moe = {"kind": "moe", "expert": {"ff": width}, "router": {"experts": 8, "top": 2}, "shared": {"ff": width}}
    return {"architecture": "Labepel", "vocab": 32000, "width": width, "max_positions": positions, "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": dict(att), "mlp": dict(moe)} for _ in range(4)]}


def hybrid_bench_config(width: int) -> Dict[str, Any]:
    h = width // 128
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 4 * width},
           "mixer": {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": min(1536, width),
                     "scale": 192 ** -0.5, "rot": {"dims": 64, "base": 10000.0}}}
    delta = {"type": "channel_delta", "mlp": {"kind": "dense", "ff": 4 * width},
             "mixer": {"heads": h, "kv_heads": max(1, h // 2), "dim": 128, "vdim": 128, "conv": 4}}
    gla = {"type": "gla", "mlp": {"kind": "dense", "ff": 4 * width}, "mixer": {"heads": h, "dim": 64, "vdim": 128, "tau": 16.0}}
    return {"architecture": "Badapel", "vocab": 32000, "width": width, "layers": [lat, delta, gla, dict(lat)],
            "norm": {"eps": 1e-6}, "logit_softcap": 30.0}


def _time(fn: Callable[[], Any], iters: int, warmup: int, flush: Any = None) -> float:
    """Median milliseconds of ``fn`` over ``iters`` runs (CUDA events; optional L2 flush between runs)."""
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(iters):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    ts.sort()
    return ts[len(ts) // 2]


def _peaks() -> Dict[str, float]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as fp:
            d = json.load(fp)
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    except (OSError, KeyError, ValueError):
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def _hybrid(width: int, prompt_len: int, batch: int, steps: int, warmup: int, design: str = "hybrid") -> Dict[str, Any]:
    from ..models.config import HybridConfig
    from ..models.hybrid import HybridLM
    from ..parallel.hybrid_runner import HybridRunner

    dev = torch.device("cuda")
    make = {"hybrid": hybrid_bench_config, "vudelix": vudelix_bench_config, "labepel": labepel_bench_config,
            "zudovik": zudovik_bench_config, "ratesun": ratesun_bench_config, "dufelix": dufelix_bench_config}[design]
    cfg = HybridConfig.from_dict(make(width))
    model = HybridLM(cfg, {}).init_random(dev, torch.bfloat16, seed=1)
    params = sum(p.numel() for p in model.tensor_map().values())
    out: Dict[str, Any] = {"params_m": round(params / 1e6, 1), "layer_params_m": round((params - model.embed.numel()) / 1e6, 1)}
    prompt = torch.randint(0, cfg.vocab, (prompt_len,)).tolist()
    S = prompt_len + steps + warmup + 8

    def prefill_once() -> None:
        r = HybridRunner(model, S, n_slots=1, use_graphs=False)
        prefill_once.r = r
        r.step([("p", prompt)])

    # the runner is rebuilt per run (a pool of zeros): its allocation is outside what a serving loop pays per
    # prompt, so time only the step by pre-building
    runners = [HybridRunner(model, S, n_slots=1, use_graphs=False) for _ in range(warmup + 5)]
    it = iter(runners)
    ms = _time(lambda: next(it).step([("p", prompt)]), 5, warmup)
    out["prefill_tok_s"] = round(prompt_len / ms * 1e3, 1)
    out["prefill_ms"] = round(ms, 3)
    del runners
    # the chunk-masked design decodes up to the end of the prompt's last chunk, not across its edge
    context = prompt if design != "labepel" else prompt[: max(1, prompt_len - steps - warmup - 8)]
    out["decode_context"] = len(context)
    for b in (1, batch):
        r = HybridRunner(model, S, n_slots=b)
        # every stream its own prompt and tokens: identical streams would all choose the same experts
        r.step([(i, torch.randint(0, cfg.vocab, (len(context),)).tolist()) for i in range(b)])
        tok = [(i, [1 + 37 * i]) for i in range(b)]
        ms = _time(lambda: r.step(tok), steps, warmup)
        out[f"decode_tok_s_b{b}"] = round(b / ms * 1e3, 1)
        out[f"decode_ms_b{b}"] = round(ms, 4)
        del r
    kernels = {"hybrid": _hybrid_kernels, "vudelix": _vudelix_kernels, "labepel": _labepel_kernels,
               "zudovik": _zudovik_kernels, "ratesun": _ratesun_kernels, "dufelix": _dufelix_kernels}[design]
    out["kernels"] = kernels(model, prompt_len, batch)
    return out


def _vudelix_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """The pre-norm design's own kernels alone, on the prompt shape and on the decode shape (see ``_hybrid_kernels``)."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt = model.device, model.dtype
    C = model.config.width
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, phase: str, ms: float, nbytes: float, flops: float) -> None:
        rows.append({"kernel": name, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    att, moe = model.blocks[1].mix, model.blocks[1].mlp
    Hh, G, D, V, W = att.H, att.G, att.D, att.V, att.window
    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [T] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        cache = pool.runs[1]["cache"]
        cache.normal_()
        h = torch.randn(N, C, device=dev).to(dt)
        p = H.linear(h, att.w_in)
        q, g = att.col(p, "q"), att.col(p, "g")
        pairs = sum(min(W, s + i + 1) if W else s + i + 1 for n, s in zip(lengths, starts) for i in range(n))
        ms = _time(lambda: H.window_append(q, att.col(p, "k"), att.col(p, "v"), att.inv_freq, cache, plan, Hh, G, D, V,
                                           att.nrot, 1e-6), 5, 3, flush)
        rec("window_append", phase, ms, 2.0 * N * (2 * Hh * D + 2 * G * (D + V)), 0.0)
        if phase == "prefill":
            ms = _time(lambda: H.head_gate(att._banded(q, cache, plan), g), 5, 3, flush)
            rec("window_attn_banded(gemm+softmax)", phase, ms, 2.0 * N * (Hh * (D + V) + G * (D + V)), 2.0 * Hh * pairs * (D + V))
            nb = min(N, att.query_block)
            s32 = torch.randn(Hh, nb, nb + W - 1, device=dev)
            ms = _time(lambda: H.causal_softmax(s32, N - nb, att.scale, dt, window=W, key0=N - nb - W + 1), 5, 3, flush)
            rec("causal_softmax[window]", phase, ms, s32.numel() * 6.0, 0.0)
            del s32
        else:
            ms = _time(lambda: H.window_attn(q, g, cache, plan, Hh, G, D, V, att.scale, W), 5, 3, flush)
            keys = sum(min(W, s + 1) if W else s + 1 for s in starts)
            rec("window_attn", phase, ms, 2.0 * G * keys * (D + V) + 2.0 * N * Hh * (D + V), 2.0 * Hh * pairs * (D + V))
        z = H.linear_f32(h, moe.router32)
        ms = _time(lambda: H.router_topk(z, moe.top), 5, 3, flush)
        rec("router_topk", phase, ms, 4.0 * N * (moe.E + 2 * moe.top), 0.0)
        ms = _time(lambda: moe(h), 5, 3, flush)
        wbytes = 2.0 * 2 * C * moe.ff * min(moe.E, N * moe.top)
        rec("moe_experts[index-driven]" if N * moe.top <= moe.gemv_max else "moe_experts[grouped gemm]", phase, ms,
            wbytes + 2.0 * N * C * (1 + moe.top), 4.0 * N * moe.top * C * moe.ff)
        ff = model.blocks[0].mlp
        ms = _time(lambda: ff(h), 5, 3, flush)
        rec("dense_ff(gemm+gelu)", phase, ms, 2.0 * 2 * C * ff.up.size(0) + 4.0 * N * C, 4.0 * N * C * ff.up.size(0))
        side = model.blocks[0].side
        zs = H.linear(h, side.gate)
        tok = torch.randint(0, model.config.vocab, (N,), device=dev, dtype=torch.int32)
        ms = _time(lambda: H.token_side_gate(zs, model.side_embed, tok, 0), 5, 3, flush)
        rec("token_side_gate", phase, ms, 2.0 * N * 3 * side.dim, 0.0)
        x = torch.randn(N, C, device=dev)
        ms = _time(lambda: H.norm_rows(x, model.blocks[0].norm1.w, None, 1e-6, "rms", dt), 5, 3, flush)
        rec("rms_norm", phase, ms, N * C * 6.0, 0.0)
        y = torch.randn(N, C, device=dev).to(dt)
        ms = _time(lambda: H.norm_accumulate(x, y, None, None, 1e-6, "none", 0.5), 5, 3, flush)
        rec("scaled_residual_add", phase, ms, N * C * 10.0, 0.0)
        del pool
    return rows


def _zudovik_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """The post-norm design's own kernels alone, on the prompt shape and on the decode shape; ``like`` names the row of
    ``_labepel_kernels`` (or, for the recurrence, of ``_hybrid_kernels``) that does the corresponding work."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt = model.device, model.dtype
    C = model.config.width
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, like: str, phase: str, ms: float, nbytes: float, flops: float) -> None:
        rows.append({"kernel": name, "like": like, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    att, lit, moe, dense = model.blocks[2].mix, model.blocks[1].mix, model.blocks[2].mlp, model.blocks[0].mlp
    Hh, G, D, V = att.H, att.G, att.D, att.V
    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [T] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        cache = pool.runs[2]["cache"]
        cache.normal_()
        tok = torch.randint(0, model.config.vocab, (N,), device=dev, dtype=torch.int32)
        ms = _time(lambda: H.embed_rows(model.embed, tok, None, plan, model.config.embed_scale), 5, 3, flush)
        rec("embed_rows[scale]", "embed_rows[positions]", phase, ms, N * C * 6.0, 0.0)
        x = torch.randn(N, C, device=dev)
        h = torch.randn(N, C, device=dev).to(dt)
        p = H.linear(h, att.w_in, att.b_in)
        q, g = att.col(p, "q"), att.col(p, "g")
        pairs = sum(s + i + 1 for n, s in zip(lengths, starts) for i in range(n))
        ms = _time(lambda: H.full_norm_append(q, att.col(p, "k"), att.col(p, "v"), att.inv_freq, cache, plan, Hh, G, D, V, att.nrot,
                                              1e-6, att.q_norm, att.k_norm), 5, 3, flush)
        rec("full_norm_append", "window_append[weights, value mixing]", phase, ms, 2.0 * N * (2 * Hh * D + 2 * G * (D + V)), 0.0)
        if phase == "prefill":
            ms = _time(lambda: H.head_gate(att._banded(q, cache, plan), g), 5, 3, flush)
            rec("causal_attn(gemm+softmax)", "chunk_attn(gemm+softmax)", phase, ms, 2.0 * N * (Hh * (D + 2 * V) + G * (D + V)),
                2.0 * Hh * pairs * (D + V))
            nb = min(N, att.query_block)
            s32 = torch.randn(Hh, nb, N, device=dev)
            ms = _time(lambda: H.causal_softmax(s32, N - nb, att.scale, dt, sink=True, split=True, cap=att.softcap,
                                                sink_vals=att.sink32), 5, 3, flush)
            rec("causal_softmax[cap, learned sink, split weights]", "causal_softmax[sink, split weights]", phase, ms,
                s32.numel() * 8.0, 0.0)
            del s32
        else:
            ms = _time(lambda: H.window_attn(q, g, cache, plan, Hh, G, D, V, att.scale, 0, sink=True, cap=att.softcap,
                                             sink_vals=att.sink32), 5, 3, flush)
            keys = sum(s + 1 for s in starts)
            rec("window_attn[causal, cap, learned sink]", "window_attn[chunk, sink, channel gate]", phase, ms,
                2.0 * G * keys * (D + V) + 2.0 * N * Hh * (D + V), 2.0 * Hh * pairs * (D + V))
        # the recurrent mixer
        LH, LD, LV = lit.H, lit.D, lit.V
        pl = H.linear(h, lit.w_in)
        state = pool.runs[1]["state"]
        ms = _time(lambda: H.lightning_recurrence(lit.col(pl, "q"), lit.col(pl, "k"), lit.col(pl, "v"), lit.decay, state,
                                                  plan, LH, LD, LV, act=True), 5, 3, flush)
        nbytes = 2.0 * N * (2 * LH * LD + LH * LV) + 4.0 * N * LH * LV + 8.0 * n_seq * LH * LD * LV
        rec("lightning_recurrence[chunks]" if phase == "prefill" else "lightning_recurrence[scan]", "gated_recurrence[gla]", phase,
            ms, nbytes, 4.0 * N * LH * LD * LV)
        o = torch.randn(N, LH * LV, device=dev)
        ms = _time(lambda: H.norm_gate_rows(o, lit.norm, lit.col(pl, "g"), 1e-6, dt), 5, 3, flush)
        rec("norm_gate_rows", "rms_norm[1 + w]", phase, ms, N * LH * LV * 8.0, 0.0)
        # feed-forwards
        z = H.linear_f32(h, moe.router32)
        ms = _time(lambda: H.router_topk(z, moe.top, "softmax_all", moe.correction32), 5, 3, flush)
        rec("router_topk[softmax over all, correction]", "router_topk[softmax]", phase, ms, 4.0 * N * (moe.E + moe.identity + 2 * moe.top), 0.0)
        ms = _time(lambda: moe(h), 5, 3, flush)
        wbytes = 2.0 * 3 * C * moe.ff * min(moe.E, N * moe.top)
        form = "index-driven" if N * moe.top <= moe.gemv_max else "grouped gemm"
        rec(f"moe_experts[{form}, clamped, identity]", f"moe_experts[{form}, gated]", phase, ms, wbytes + 2.0 * N * C * (1 + moe.top),
            6.0 * N * moe.top * C * moe.ff)
        sh = moe.shared
        ms = _time(lambda: sh.gated(h), 5, 3, flush)
        rec("shared_expert(gemm+clamped product)", "shared_expert(gemm+silu*up)", phase, ms, 2.0 * 3 * C * sh.ff + 4.0 * N * C,
            6.0 * N * C * sh.ff)
        gu = H.linear(h, sh.w_in)
        ms = _time(lambda: H.act_mul(gu[:, :2 * sh.ff], "clamped", sh.limit), 5, 3, flush)
        rec("act_mul[clamped]", "act_mul", phase, ms, 2.0 * N * 3 * sh.ff, 0.0)
        ms = _time(lambda: dense(h), 5, 3, flush)
        rec("dense_ff(gemm+relu2)", "shared_expert(gemm+silu*up)", phase, ms, 2.0 * 2 * C * dense.up.size(0) + 4.0 * N * C,
            4.0 * N * C * dense.up.size(0))
        ya, yb = (torch.randn(N, C, device=dev).to(dt) for _ in range(2))
        sg = torch.randn(N, 1, device=dev).to(dt)
        blk = model.blocks[2]
        cp = torch.empty(N, C, device=dev, dtype=dt)
        ms = _time(lambda: H.norm_accumulate(x, ya, blk.norm1.w, None, 1e-6, "rms", copy=cp), 5, 3, flush)
        rec("post_norm_accumulate[+ rounded copy]", "scaled_branches", phase, ms, N * C * 12.0, 0.0)
        ms = _time(lambda: H.gated_sum_norm_accumulate(x, ya, yb, sg, blk.norm2.w, 1e-6, copy=cp), 5, 3, flush)
        rec("gated_sum_norm_accumulate[+ rounded copy]", "scaled_branches", phase, ms, N * C * 14.0, 0.0)
        del pool
    return rows


def _ratesun_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """The kernels of the sandwich design with input convolutions and an average over depth; ``like`` names the row of
    ``_hybrid_kernels`` (or, for the per-layer token embedding, of ``_vudelix_kernels``) that does the corresponding work."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt, cfg = model.device, model.dtype, model.config
    C = cfg.width
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, like: str, phase: str, fn: Callable[[], Any], nbytes: float, flops: float = 0.0) -> None:
        ms = _time(fn, 5, 3, flush)
        rows.append({"kernel": name, "like": like, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    blk = model.blocks[2]
    mix, side, taps, bg = blk.mix, blk.side, cfg.canon_taps, cfg.bigram
    Hh, D, R, V, L, W = mix.H, mix.D, mix.R, mix.V, mix.L, mix.window
    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [T] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        st = pool.runs[2]
        st["cache"].normal_()
        tok = torch.randint(0, cfg.vocab, (N,), device=dev, dtype=torch.int32)
        depth = torch.randn(6, N, C, device=dev)
        x, y = depth[3], torch.randn(N, C, device=dev).to(dt)
        b1 = (blk.norm1b.w, blk.norm1b.b, 1e-6, "layer", 0.5)
        conv_bytes = 8.0 * n_seq * (taps - 1) * C  # state read and written
        rec("embed_pairs", "embed_rows", phase,
            lambda: H.embed_pairs(model.embed, model.bigram, tok, plan, pool.prev, bg["buckets"], bg["mul_prev"], bg["mul_cur"], 1.0,
                                  depth[0], depth[1]), N * C * 12.0)
        if phase == "prefill":
            rec("norm_conv", "layer_norm", phase, lambda: H.norm_conv(x, blk._input1(st), plan, dt), N * C * 6.0 + conv_bytes)
            rec("row_update", "norm_accumulate", phase, lambda: H.row_update(x, y, *b1), N * C * 10.0)
            rec("row_update[depth average of 4 rows]", "norm_accumulate", phase,
                lambda: H.row_update(x, y, side.norm, None, 1e-6, "rms", 0.5, depth=depth, index=3, depth_w=blk.depth_w), N * C * 26.0)
        else:
            rec("row_update[+ next norm, convolution]", "norm_accumulate", phase,
                lambda: H.row_update(x, y, *b1, nxt=blk._input2(st), plan=plan, out_dtype=dt), N * C * 12.0 + conv_bytes)
            rec("row_update[depth average, next norm, convolution]", "norm_accumulate", phase,
                lambda: H.row_update(x, y, side.norm, None, 1e-6, "rms", 0.5, depth=depth, index=3, depth_w=blk.depth_w,
                                     nxt=blk._input1(st), plan=plan, out_dtype=dt), N * C * 28.0 + conv_bytes)
        h = torch.randn(N, C, device=dev).to(dt)
        p = H.linear(h, mix.w_in)
        rec("latent_prepare", "latent_prepare", phase,
            lambda: H.latent_prepare(mix.col(p, "dq"), mix.dq_norm, mix.col(p, "dkv"), mix.dkv_norm, mix.inv_freq, st["cache"], plan, R, L,
                                     mix.nrot, 1e-6, mix.pairing), 4.0 * N * (L + R + mix.QR))
        q = H.linear(h[:, :mix.QR].contiguous(), mix.uq)
        keys = sum(min(W, s + i + 1) for n, s in zip(lengths, starts) for i in range(n))  # visible (query, key) pairs
        if phase == "prefill":
            rec("rotate_heads", "latent_prepare", phase,
                lambda: H.rotate_heads(q, mix.inv_freq, plan, Hh, D, R, mix.nrot, mix.pairing), 4.0 * N * Hh * R)
            rec("latent_attn_expanded[window]", "latent_attn_expanded", phase, lambda: mix._expanded(q, st["cache"], plan),
                2.0 * N * Hh * (D + R + V), 2.0 * T * L * Hh * (D + V) + 2.0 * Hh * keys * (D + R + V))
        else:
            qlat = torch.randn(Hh, N, L, device=dev)
            rec("latent_attn[window, rotation]", "latent_attn", phase,
                lambda: H.latent_attn(qlat, q, st["cache"], plan, Hh, D, R, L, mix.scale, window=W, inv_freq=mix.inv_freq, nrot=mix.nrot,
                                      pairing=mix.pairing),
                6.0 * Hh * N * L + 2.0 * Hh * N * R + 2.0 * (L + R) * sum(min(W, s + 1) for s in starts), 2.0 * Hh * keys * (2 * L + R))
        a = torch.randn(N, blk.mlp.up.size(0), device=dev).to(dt)
        rec("poly_norm", "gelu", phase, lambda: H.poly_norm(a, blk.mlp.coef32, 1e-6), 4.0 * a.numel())
        rec("dense_ff(gemm+poly_norm)", "dense_ff(gemm+gelu)", phase, lambda: blk.mlp(h), 4.0 * C * a.size(1) + 4.0 * N * C,
            4.0 * N * C * a.size(1))
        zs = H.linear(h, side.gate)
        rec("token_side_gate", "token_side_gate", phase, lambda: H.token_side_gate(zs, model.side_embed, tok, 0), 6.0 * N * side.dim)
        del pool
    return rows


def _dufelix_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """The RMS sandwich design's kernels alone; ``like`` names the row of ``_ratesun_kernels`` (or of ``_zudovik_kernels`` for the
    grouped-query attention, the recurrence and its norm, of ``_hybrid_kernels`` for the convolution) with the corresponding work."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt, cfg = model.device, model.dtype, model.config
    C = cfg.width
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, like: str, phase: str, fn: Callable[[], Any], nbytes: float, flops: float = 0.0) -> None:
        ms = _time(fn, 5, 3, flush)
        rows.append({"kernel": name, "like": like, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    blk, att, lat, ssm = model.blocks[0], model.blocks[0].mix, model.blocks[1].mix, model.blocks[2].mix
    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [T] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        pool.runs[0]["cache"].normal_()
        pool.runs[1]["cache"].normal_()
        pairs = sum(s + i + 1 for n, s in zip(lengths, starts) for i in range(n))  # visible (query, key) pairs
        keys = sum(s + n for n, s in zip(lengths, starts))
        x, y, h = torch.randn(N, C, device=dev), torch.randn(N, C, device=dev).to(dt), torch.randn(N, C, device=dev).to(dt)
        tok = torch.randint(0, cfg.vocab, (N,), device=dev, dtype=torch.int32)
        rec("embed_rows[scale]", "embed_rows[scale]", phase, lambda: H.embed_rows(model.embed, tok, None, plan, cfg.embed_scale), N * C * 6.0)
        rec("row_update[rms, + next norm]", "row_update" if phase == "prefill" else "row_update[+ next norm, convolution]", phase,
            lambda: H.row_update(x, y, blk.norm1b.w, None, 1e-6, "rms", nxt=blk._input2({}), plan=plan, out_dtype=dt), N * C * 12.0)
        # grouped-query attention
        Hh, G, D, V = att.H, att.G, att.D, att.V
        cache = pool.runs[0]["cache"]
        p = H.linear(h, att.w_in)
        q, g = att.col(p, "q"), att.col(p, "g")
        rec("window_append[halves, no norm]", "full_norm_append", phase,
            lambda: H.window_append(q, att.col(p, "k"), att.col(p, "v"), att.inv_freq, cache, plan, Hh, G, D, V, att.nrot, 1e-6, norm=False,
                                    pairing=att.pairing, amp=att.amp), 2.0 * N * (2 * Hh * D + 2 * G * (D + V)))
        if phase == "prefill":
            rec("grouped_attn[fused, gate]", "causal_attn(gemm+softmax)", phase, lambda: att._fused(q, g, cache, plan),
                2.0 * N * (Hh * (D + V) + G * (D + V)), 2.0 * Hh * pairs * (D + V))
        else:
            rec("window_attn[causal, gate]", "window_attn[causal, cap, learned sink]", phase,
                lambda: H.window_attn(q, g, cache, plan, Hh, G, D, V, att.scale, 0),
                2.0 * G * keys * (D + V) + 2.0 * N * Hh * (D + V), 2.0 * Hh * pairs * (D + V))
        # latent attention
        Hh, D, R, V, L = lat.H, lat.D, lat.R, lat.V, lat.L
        cache = pool.runs[1]["cache"]
        p = H.linear(h, lat.w_in)
        rec("latent_prepare", "latent_prepare", phase,
            lambda: H.latent_prepare(lat.col(p, "dq"), lat.dq_norm, lat.col(p, "dkv"), lat.dkv_norm, lat.inv_freq, cache, plan, R, L,
                                     lat.nrot, 1e-6, lat.pairing, lat.amp), 4.0 * N * (L + R + lat.QR))
        q = H.linear(h[:, :lat.QR].contiguous(), lat.uq)
        if phase == "prefill":
            rec("rotate_heads", "rotate_heads", phase,
                lambda: H.rotate_heads(q, lat.inv_freq, plan, Hh, D, R, lat.nrot, lat.pairing, lat.amp), 4.0 * N * Hh * R)
            rec("latent_attn_expanded[sink]", "latent_attn_expanded[window]", phase, lambda: lat._expanded(q, cache, plan),
                2.0 * N * Hh * (D + R + V), 2.0 * T * L * Hh * (D + V) + 2.0 * Hh * pairs * (D + R + V))
        else:
            qlat = torch.randn(Hh, N, L, device=dev)
            rec("latent_attn[sink, rotation]", "latent_attn[window, rotation]", phase,
                lambda: H.latent_attn(qlat, q, cache, plan, Hh, D, R, L, lat.scale, inv_freq=lat.inv_freq, nrot=lat.nrot,
                                      pairing=lat.pairing, amp=lat.amp, sink=lat.sink32),
                6.0 * Hh * N * L + 2.0 * Hh * N * R + 2.0 * (L + R) * keys, 2.0 * Hh * pairs * (2 * L + R))
        # the recurrence
        Hh, V, S, G, a, b = ssm.H, ssm.V, ssm.N, ssm.G, ssm.inner, ssm.inner + ssm.ch
        st = pool.runs[2]
        p = H.linear(h, ssm.w_in)
        rec("conv_silu[bias]", "conv_silu", phase, lambda: H.conv_silu(p[:, a:b], ssm.conv, st["conv"], plan, ssm.conv_b), 4.0 * N * ssm.ch)
        xbc = H.conv_silu(p[:, a:b], ssm.conv, st["conv"], plan, ssm.conv_b)
        rec("ssd_recurrence[chunks]" if phase == "prefill" else "ssd_recurrence[scan]",
            "lightning_recurrence[chunks]" if phase == "prefill" else "lightning_recurrence[scan]", phase,
            lambda: H.ssd_recurrence(xbc, p[:, b:b + Hh], ssm.dt_bias32, ssm.A_log32, ssm.skip32, st["state"], plan, Hh, G, S, V),
            2.0 * N * (ssm.ch + Hh) + 4.0 * N * a + 8.0 * n_seq * Hh * S * V, 4.0 * N * Hh * S * V)
        o = torch.randn(N, a, device=dev)
        rec("silu_gate_norm[parts]", "norm_gate_rows", phase, lambda: H.silu_gate_norm(o, p[:, :a], ssm.norm, ssm.parts, 1e-6, dt), N * a * 8.0)
        ff = blk.mlp
        gu = H.linear(h, ff.w_in)
        rec("act_mul[gelu]", "act_mul[clamped]", phase, lambda: H.act_mul(gu, "gelu_tanh"), 6.0 * N * ff.ff)
        rec("dense_ff(gemm+gelu*up)", "dense_ff(gemm+poly_norm)", phase, lambda: ff(h), 6.0 * C * ff.ff + 4.0 * N * C, 6.0 * N * C * ff.ff)
        del pool
    return rows


def _labepel_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """The parallel-block design's own kernels alone, on the prompt shape and on the decode shape; ``like`` names the
    row of ``_vudelix_kernels`` that does the corresponding work in the pre-norm design."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt = model.device, model.dtype
    C = model.config.width
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, like: str, phase: str, ms: float, nbytes: float, flops: float) -> None:
        rows.append({"kernel": name, "like": like, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    blk = model.blocks[1]  # a layer that blends its values with the first layer's
    att, moe = blk.mix, blk.mlp
    Hh, G, D, V, W = att.H, att.G, att.D, att.V, att.window
    first = lambda pos: (pos // W) * W if W else 0  # noqa: E731 - first visible key of a position
    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [max(0, T - 8)] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        cache = pool.runs[1]["cache"]
        cache.normal_()
        tok = torch.randint(0, model.config.vocab, (N,), device=dev, dtype=torch.int32)
        ms = _time(lambda: H.embed_rows(model.embed, tok, model.pos, plan), 5, 3, flush)
        rec("embed_rows[positions]", "", phase, ms, N * C * 8.0, 0.0)
        h = torch.randn(N, C, device=dev).to(dt)
        p = H.linear(h, att.w_in, att.b_in)
        q, g, v = att.col(p, "q"), att.col(p, "g"), att.col(p, "v")
        vf = torch.randn_like(v)
        pairs = sum(s + i + 1 - first(s + i) for n, s in zip(lengths, starts) for i in range(n))
        ms = _time(lambda: H.window_append(q, att.col(p, "k"), v, None, cache, plan, Hh, G, D, V, 0, 1e-6, att.q_norm,
                                           att.k_norm, vf, att.lam), 5, 3, flush)
        rec("window_append[weights, value mixing]", "window_append", phase, ms,
            2.0 * N * (2 * Hh * D + 2 * G * (D + V) + G * V), 0.0)
        if phase == "prefill":
            ms = _time(lambda: H.headmajor_gate(att._chunked(q, cache, plan), g), 5, 3, flush)
            rec("chunk_attn(gemm+softmax)", "window_attn_banded(gemm+softmax)", phase, ms,
                2.0 * N * (Hh * (D + 2 * V) + G * (D + V)), 2.0 * Hh * pairs * (D + V))
            nb = min(N, W) if W else min(N, att.query_block)
            s32 = torch.randn(max(1, N // nb) * Hh, nb, nb, device=dev)
            ms = _time(lambda: H.causal_softmax(s32, 0, att.scale, dt, sink=att.sink, split=True), 5, 3, flush)
            rec("causal_softmax[sink, split weights]", "causal_softmax[window]", phase, ms, s32.numel() * 8.0, 0.0)
            del s32
        else:
            ms = _time(lambda: H.window_attn(q, g, cache, plan, Hh, G, D, V, att.scale, W, mask=att.mask_kind, sink=att.sink),
                       5, 3, flush)
            keys = sum(s + 1 - first(s) for s in starts)
            rec("window_attn[chunk, sink, channel gate]", "window_attn", phase, ms,
                2.0 * G * keys * (D + V) + 2.0 * N * Hh * (D + 2 * V), 2.0 * Hh * pairs * (D + V))
        z = H.linear_f32(h, moe.router32, moe.router_b32)
        ms = _time(lambda: H.router_topk(z, moe.top, "softmax"), 5, 3, flush)
        rec("router_topk[softmax]", "router_topk", phase, ms, 4.0 * N * (moe.E + 2 * moe.top), 0.0)
        ms = _time(lambda: moe(h), 5, 3, flush)
        wbytes = 2.0 * 3 * C * moe.ff * min(moe.E, N * moe.top)
        form = "index-driven" if N * moe.top <= moe.gemv_max else "grouped gemm"
        rec(f"moe_experts[{form}, gated]", f"moe_experts[{form}]", phase, ms, wbytes + 2.0 * N * C * (1 + moe.top),
            6.0 * N * moe.top * C * moe.ff)
        sh = moe.shared
        ms = _time(lambda: sh(h), 5, 3, flush)
        rec("shared_expert(gemm+silu*up)", "dense_ff(gemm+gelu)", phase, ms, 2.0 * 3 * C * sh.down.size(1) + 4.0 * N * C,
            6.0 * N * C * sh.down.size(1))
        gu = H.linear(h, sh.w_in)
        ms = _time(lambda: H.act_mul(gu), 5, 3, flush)
        rec("act_mul", "", phase, ms, 2.0 * N * 3 * sh.down.size(1), 0.0)
        x = torch.randn(N, C, device=dev)
        ms = _time(lambda: H.norm_rows(x, blk.norm1.w, None, 1e-6, "rms", dt, 1.0), 5, 3, flush)
        rec("rms_norm[1 + w]", "rms_norm", phase, ms, N * C * 6.0, 0.0)
        ya, yb, yc = (torch.randn(N, C, device=dev).to(dt) for _ in range(3))
        ms = _time(lambda: H.scaled_branches(x, ya, blk.ls1, yb, yc, blk.ls2), 5, 3, flush)
        rec("scaled_branches", "scaled_residual_add", phase, ms, N * C * 14.0, 0.0)
        del pool
    return rows


def _hybrid_kernels(model: Any, T: int, batch: int) -> List[Dict[str, Any]]:
    """Each family kernel alone, on the prompt shape (1 x T tokens) and the decode shape (batch x 1 token at context T)."""
    from ..ops import hybrid as H

    pk = _peaks()
    dev, dt = model.device, model.dtype
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict[str, Any]] = []

    def rec(name: str, phase: str, ms: float, nbytes: float, flops: float) -> None:
        rows.append({"kernel": name, "phase": phase, "ms": round(ms, 4), "gb_s": round(nbytes / ms / 1e6, 1),
                     "tflops": round(flops / ms / 1e9, 2),
                     "frac_of_roofline": round(max(nbytes / ms / 1e6 / pk["hbm_gbs"], flops / ms / 1e9 / pk["bf16_tflops"]), 4),
                     "peaks": pk["source"]})

    for phase, lengths, starts in (("prefill", [T], [0]), ("decode", [1] * batch, [T] * batch)):
        n_seq, N = len(lengths), sum(lengths)
        pool = model.new_pool(n_seq, T + 8)
        plan = H.BatchPlan.make(lengths, list(range(n_seq)), starts, dev)
        for li, blk in enumerate(model.blocks[:3]):
            mix, st = blk.mix, pool.runs[li]
            h = torch.randn(N, model.config.width, device=dev).to(dt)
            p = H.linear(h, mix.w_in)
            if li == 0:
                Hh, D, R, V, L = mix.H, mix.D, mix.R, mix.V, mix.L
                st["cache"].normal_()
                q = H.linear(H.norm_rows(mix.col(p, "dq"), mix.dq_norm, None, 1e-6, "rms", dt), mix.uq)
                qlat = torch.randn(Hh, N, L, device=dev).to(dt)
                keys = sum((s + n) * n - n * (n - 1) // 2 for n, s in zip(lengths, starts))  # visible (query, key) pairs
                if phase == "prefill":  # prompts take the expanded form: GEMMs + the causal softmax kernel
                    ms = _time(lambda: mix._expanded(q, st["cache"], plan), 5, 3, flush)
                    total_keys = sum(s + n for n, s in zip(lengths, starts))
                    flops = 2.0 * total_keys * L * Hh * (D + V) + 2.0 * Hh * keys * (D + R + V)
                    rec("latent_attn_expanded", phase, ms, 2.0 * N * Hh * (D + R + V), flops)
                    s32 = torch.randn(Hh, min(N, 1024), N, device=dev)
                    ms = _time(lambda: H.causal_softmax(s32, N - s32.size(1), mix.scale, dt), 5, 3, flush)
                    rec("causal_softmax", phase, ms, s32.numel() * 6.0, 0.0)
                    del s32
                else:
                    ms = _time(lambda: H.latent_attn(qlat, q, st["cache"], plan, Hh, D, R, L, mix.scale), 5, 3, flush)
                    nbytes = 2.0 * (2 * Hh * N * L + Hh * N * R) + 2.0 * (L + R) * sum(s + n for n, s in zip(lengths, starts))
                    rec("latent_attn", phase, ms, nbytes, 2.0 * Hh * keys * (2 * L + R))
                ms = _time(lambda: H.latent_prepare(mix.col(p, "dq"), mix.dq_norm, mix.col(p, "dkv"), mix.dkv_norm, mix.inv_freq,
                                                    st["cache"], plan, R, L, mix.nrot, 1e-6), 5, 3, flush)
                rec("latent_prepare", phase, ms, 4.0 * N * (L + R + mix.QR), 0.0)
            else:
                mode = "delta" if li == 1 else "gla"
                Hh, D, V = mix.H, mix.D, mix.V
                G = mix.G if mode == "delta" else Hh
                z = torch.randn(N, Hh * D, device=dev).to(dt)
                gate = torch.randn(N, Hh * V, device=dev).to(dt)
                if mode == "delta":
                    c = H.conv_silu(p[:, :2 * G * D + Hh * V], mix.conv_w, st["conv"], plan)
                    args = (c[:, :G * D], c[:, G * D:2 * G * D], c[:, 2 * G * D:], z, gate, mix.norm, st["state"], plan)
                    kw = dict(heads=Hh, kv_heads=G, dim=D, vdim=V, mode=mode, eps=1e-6, zb=mix.dt_bias, beta=mix.col(p, "b"),
                              a_log=mix.A_log)
                    ms = _time(lambda: H.conv_silu(p[:, :2 * G * D + Hh * V], mix.conv_w, st["conv"], plan), 5, 3, flush)
                    rec("conv_silu", phase, ms, 2.0 * N * 2 * (2 * G * D + Hh * V), 0.0)
                else:
                    args = (mix.col(p, "q"), mix.col(p, "k"), mix.col(p, "v"), z, gate, mix.norm, st["state"], plan)
                    kw = dict(heads=Hh, kv_heads=G, dim=D, vdim=V, mode=mode, eps=1e-6, zb=mix.a2_b, tau=mix.tau)
                ms = _time(lambda: H.gated_recurrence(*args, **kw), 5, 3, flush)
                nbytes = 2.0 * N * (2 * G * D + Hh * D + 3 * Hh * V) + 8.0 * n_seq * Hh * D * V
                rec(f"gated_recurrence[{mode}]", phase, ms, nbytes, (6.0 if mode == "delta" else 4.0) * N * Hh * D * V)
        x = torch.randn(N, model.config.width, device=dev)
        blk = model.blocks[0]
        ms = _time(lambda: H.norm_rows(x, blk.norm1.w, blk.norm1.b, 1e-6, "layer", dt), 5, 3, flush)
        rec("layer_norm", phase, ms, N * model.config.width * 6.0, 0.0)
        C = model.config.width
        y = torch.randn(N, C, device=dev).to(dt)
        ms = _time(lambda: H.norm_accumulate(x, y, blk.norm1b.w, blk.norm1b.b, 1e-6), 5, 3, flush)
        rec("norm_accumulate", phase, ms, N * C * 10.0, 0.0)
        tok = torch.randint(0, model.config.vocab, (N,), device=dev, dtype=torch.int32)
        ms = _time(lambda: H.embed_rows(model.embed, tok), 5, 3, flush)
        rec("embed_rows", phase, ms, N * C * 6.0, 0.0)
        a = torch.randn(N, blk.mlp.up.size(0), device=dev).to(dt)
        ms = _time(lambda: H.gelu_(a), 5, 3, flush)
        rec("gelu", phase, ms, 4.0 * a.numel(), 0.0)
        ms = _time(lambda: blk.mlp(y), 5, 3, flush)
        rec("dense_ff(gemm+gelu)", phase, ms, 4.0 * C * a.size(1) + 4.0 * N * C, 4.0 * N * C * a.size(1))
        del pool
    return rows


def _transformer(width: int, prompt_len: int, steps: int, warmup: int, target_params: float) -> Dict[str, Any]:
    from ..models.config import Config
    from ..models.stage import build_stage
    from ..parallel.pipeline import DevicePipeline
    from ..parallel.scheduler import SamplingParams
    from ..utils.checkpoint import random_init_stage_

    n_head = width // 128
    groups = 8 if n_head % 8 == 0 else n_head
    attn = width * (n_head + 2 * groups) * 128 + width * width
    inter = int(max(256, round((target_params / 4 - attn) / (3 * width) / 256) * 256))  # equal parameters per layer
    cfg = Config(name="Llama-like-bench", block_size=prompt_len + steps + warmup + 64, vocab_size=32000, padded_vocab_size=32000,
                 n_layer=4, n_head=n_head, n_embd=width, n_query_groups=groups, rotary_percentage=1.0, parallel_residual=False,
                 bias=False, norm_class_name="RMSNorm", mlp_class_name="LLaMAMLP", intermediate_size=inter)
    stage = build_stage(cfg, "starter", cfg.n_layer, meta=True)
    random_init_stage_(stage, "cuda", torch.bfloat16)
    params = sum(p.numel() for p in stage.parameters())
    S = cfg.block_size
    pipe = DevicePipeline(stage, 0, 1, n_samples=1, max_seq_length=S, sampling=SamplingParams.greedy(), max_prompt_len=prompt_len)
    prompt = torch.randint(0, 32000, (prompt_len,), dtype=torch.int32)
    layer_params = sum(p.numel() for p in stage.transformer.h.parameters())
    out: Dict[str, Any] = {"params_m": round(params / 1e6, 1), "layer_params_m": round(layer_params / 1e6, 1), "intermediate_size": inter}

    def pre() -> None:
        pipe.prepare([prompt], steps + warmup + 8)
        torch.cuda.synchronize()

    ts = []
    for i in range(warmup + 5):
        pre()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        pipe.prefill()
        b.record()
        torch.cuda.synchronize()
        if i >= warmup:
            ts.append(a.elapsed_time(b))
    ts.sort()
    ms = ts[len(ts) // 2]
    out["prefill_tok_s"] = round(prompt_len / ms * 1e3, 1)
    out["prefill_ms"] = round(ms, 3)
    pipe.decode_rounds(warmup)
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    pipe.decode_rounds(steps)
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / steps
    out["decode_tok_s_b1"] = round(1e3 / ms, 1)
    out["decode_ms_b1"] = round(ms, 4)
    pipe.close()
    return out


def run_family_compare(widths: List[int], prompt_len: int = 2048, batch: int = 8, steps: int = 64, warmup: int = 8,
                       family: str = "hybrid") -> Dict[str, Any]:
    torch.backends.cuda.matmul.allow_tf32 = False
    results = []
    if family == "vudelix":
        for w in widths:
            new = _hybrid(w, prompt_len, batch, steps, warmup, "vudelix")
            torch.cuda.empty_cache()
            old = _hybrid(w, prompt_len, batch, steps, warmup, "hybrid")
            torch.cuda.empty_cache()
            results.append({"width": w, "vudelix": new, "hybrid": old})
        return {"metric": "family_compare", "family": "vudelix", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
                "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
                "results": results}
    if family == "zudovik":
        from ..models.config import HybridConfig
        from ..models.hybrid import HybridLM

        for w in widths:
            new = _hybrid(w, prompt_len, batch, steps, warmup, "zudovik")
            torch.cuda.empty_cache()
            old = _hybrid(w, prompt_len, batch, steps, warmup, "labepel")
            torch.cuda.empty_cache()
            # the recurrence's like kernel lives in the sandwich design: its kernels alone, no model-level timing
            sandwich = HybridLM(HybridConfig.from_dict(hybrid_bench_config(w)), {}).init_random(torch.device("cuda"), torch.bfloat16, seed=1)
            rec_rows = [k for k in _hybrid_kernels(sandwich, prompt_len, batch) if k["kernel"] == "gated_recurrence[gla]"]
            del sandwich
            torch.cuda.empty_cache()
            theirs = {(k["kernel"], k["phase"]): k["frac_of_roofline"] for k in old["kernels"] + rec_rows}
            for k in new["kernels"]:  # how far from its roofline, relative to the like kernel (above 1: this one is nearer)
                other = theirs.get((k["like"], k["phase"]))
                k["roofline_vs_like"] = round(k["frac_of_roofline"] / other, 3) if other else None
            results.append({"width": w, "zudovik": new, "labepel": old, "sandwich_recurrence": rec_rows})
        return {"metric": "family_compare", "family": "zudovik", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
                "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
                "results": results}
    if family == "ratesun":
        from ..models.config import HybridConfig
        from ..models.hybrid import HybridLM

        for w in widths:
            new = _hybrid(w, prompt_len, batch, steps, warmup, "ratesun")
            torch.cuda.empty_cache()
            old = _hybrid(w, prompt_len, batch, steps, warmup, "hybrid")
            torch.cuda.empty_cache()
            # the per-layer token embedding's like kernel lives in the pre-norm design: its kernels alone
            prenorm = HybridLM(HybridConfig.from_dict(vudelix_bench_config(w)), {}).init_random(torch.device("cuda"), torch.bfloat16, seed=1)
            side_rows = [k for k in _vudelix_kernels(prenorm, prompt_len, batch) if k["kernel"] == "token_side_gate"]
            del prenorm
            torch.cuda.empty_cache()
            theirs = {(k["kernel"], k["phase"]): k for k in old["kernels"] + side_rows}
            for k in new["kernels"]:  # how far from its roofline, relative to the like kernel (above 1: this one is nearer)
                other = theirs.get((k["like"], k["phase"]))
                k["like_ms"] = other["ms"] if other else None
                k["roofline_vs_like"] = round(k["frac_of_roofline"] / other["frac_of_roofline"], 3) \
                    if other and other["frac_of_roofline"] else None
            results.append({"width": w, "ratesun": new, "hybrid": old, "prenorm_side": side_rows})
        return {"metric": "family_compare", "family": "ratesun", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
                "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
                "results": results}
    if family == "dufelix":
        from ..models.config import HybridConfig
        from ..models.hybrid import HybridLM

        for w in widths:
            new = _hybrid(w, prompt_len, batch, steps, warmup, "dufelix")
            torch.cuda.empty_cache()
            old = _hybrid(w, prompt_len, batch, steps, warmup, "ratesun")
            torch.cuda.empty_cache()
            theirs = {(k["kernel"], k["phase"]): k for k in old["kernels"]}
            others: List[Dict[str, Any]] = []  # like kernels of designs that are not timed as a whole here
            for make, rows_of in ((zudovik_bench_config, _zudovik_kernels), (hybrid_bench_config, _hybrid_kernels)):
                model = HybridLM(HybridConfig.from_dict(make(w)), {}).init_random(torch.device("cuda"), torch.bfloat16, seed=1)
                wanted = {k["like"] for k in new["kernels"]}
                others += [k for k in rows_of(model, prompt_len, batch) if k["kernel"] in wanted and (k["kernel"], k["phase"]) not in theirs]
                theirs.update({(k["kernel"], k["phase"]): k for k in others})
                del model
                torch.cuda.empty_cache()
            for k in new["kernels"]:  # how far from its roofline, relative to the like kernel (above 1: this one is nearer)
                other = theirs.get((k["like"], k["phase"]))
                k["like_ms"] = other["ms"] if other else None
                k["roofline_vs_like"] = round(k["frac_of_roofline"] / other["frac_of_roofline"], 3) \
                    if other and other["frac_of_roofline"] else None
            results.append({"width": w, "dufelix": new, "ratesun": old, "like_kernels": others})
        return {"metric": "family_compare", "family": "dufelix", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
                "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
                "results": results}
    if family == "labepel":
        for w in widths:
            new = _hybrid(w, prompt_len, batch, steps, warmup, "labepel")
            torch.cuda.empty_cache()
            old = _hybrid(w, prompt_len, batch, steps, warmup, "vudelix")
            torch.cuda.empty_cache()
            theirs = {(k["kernel"], k["phase"]): k["frac_of_roofline"] for k in old["kernels"]}
            for k in new["kernels"]:  # how far from its roofline, relative to the like kernel of the other design
                other = theirs.get((k["like"], k["phase"]))
                k["roofline_vs_like"] = round(k["frac_of_roofline"] / other, 3) if other else None
            results.append({"width": w, "labepel": new, "vudelix": old})
        return {"metric": "family_compare", "family": "labepel", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
                "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
                "results": results}
    for w in widths:
        hy = _hybrid(w, prompt_len, batch, steps, warmup)
        torch.cuda.empty_cache()
        try:
            tr = _transformer(w, prompt_len, steps, warmup, hy["layer_params_m"] * 1e6)
        except Exception as e:  # noqa: BLE001 - the comparison arm must not hide the family's own numbers
            tr = {"error": f"{type(e).__name__}: {e}"}
        torch.cuda.empty_cache()
        results.append({"width": w, "hybrid": hy, "transformer": tr})
    return {"metric": "family_compare", "family": "hybrid", "dtype": "bf16", "data": "synthetic", "prompt_len": prompt_len,
            "decode_batch": batch, "steps": steps, "warmup": warmup, "l2": "flushed between single-kernel timings",
            "results": results}
