"""The Dufelix design (sandwich blocks with RMS norms over grouped-query attention, latent attention with sinks and a
state-space recurrence, stretched rotations, layers that share weights) against the plain oracle of ``dufelix_oracle.py``.

Every test builds its own small configuration with random weights.  Sizes are awkward on purpose: value width != key
width, odd heads and head sizes beside ones in whole 16-byte groups, partly rotated heads, one to five convolution taps,
one group or as many as heads, norms in one part or several, layers without feed-forward.  The same tests run on the CPU
(PyTorch bodies of the operations) and, marked ``gpu``, on the sm_100a kernels.
"""
from __future__ import annotations

import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import dufelix_oracle as O
from mdi_llm_b200.models.config import HybridConfig
from mdi_llm_b200.models.hybrid import GatedFF, HybridLM, LatentAttention, WindowAttention, load_hybrid, write_safetensors
from mdi_llm_b200.models.registry import model_classes
from mdi_llm_b200.ops import hybrid as H
from mdi_llm_b200.ops.hybrid import BatchPlan
from mdi_llm_b200.parallel.hybrid_runner import HybridRunner
from mdi_llm_b200.parallel.scheduler import SamplingParams

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def yarn(factor=4.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def att(heads=6, kv=3, dim=10, vdim=7, scale=0.4, rot=6, base=300.0, scaling="yarn", ff=18):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = yarn() if scaling == "yarn" else scaling
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": r}}


def lat(heads=3, dim=10, rot=6, vdim=7, kv=14, qr=11, scale=0.3, base=500.0, scaling="yarn", ff=20):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = yarn(2.0, 128, 16.0, 2.0) if scaling == "yarn" else scaling
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv, "q_rank": qr, "scale": scale, "rot": r}}


def ssm(heads=4, vdim=6, state=9, groups=2, conv=4, parts=3, ff=14):
    return {"type": "mamba2", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": parts}}


def same_as(j, entry):
    return {**copy.deepcopy(entry), "weights_of": j}


def cfg_dict(layers, width=22, vocab=50, eps=1e-3, scale=3.0):
    return {"architecture": "Dufelix", "vocab": vocab, "width": width, "layers": copy.deepcopy(layers), "norm": {"eps": eps},
            "embedding": {"scale": scale}}


# odd sizes, every mixer, repeats of each, a layer without feed-forward, two repeats of one layer; and sizes in whole 16-byte groups
BASE = [ssm(), att(), lat(), ssm(heads=2, vdim=5, state=4, groups=1, conv=2, parts=1, ff=0)]
FULL = cfg_dict(BASE + [same_as(1, BASE[1]), same_as(0, BASE[0]), same_as(2, BASE[2]), same_as(3, BASE[3]), same_as(1, BASE[1])])
BASE32 = [lat(heads=5, dim=16, rot=16, vdim=16, kv=32, qr=24, ff=48), ssm(heads=4, vdim=16, state=32, groups=2, parts=2, ff=32),
          att(heads=8, kv=2, dim=32, vdim=16, rot=16, scale=0.2, ff=40), ssm(heads=3, vdim=24, state=16, groups=3, conv=3, parts=3, ff=0)]
FULL32 = cfg_dict(BASE32 + [same_as(1, BASE32[1]), same_as(2, BASE32[2]), same_as(0, BASE32[0])], width=48, eps=1e-5, scale=7.0)

DEVICES = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
           pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]
WHERE = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]
DTYPES = [torch.float32, torch.bfloat16]


def build(d, dev, seed=0):
    device, dtype = dev
    if device == "cuda":
        torch.backends.cuda.matmul.allow_tf32 = False
    return HybridLM(HybridConfig.from_dict(d)).load_tensors(O.random_tensors(d, seed), device, dtype)


def oracle_logits(d, model, tokens, trace=None):
    W = {k: v.detach().float().cpu() for k, v in model.state_tensors().items()}
    return O.forward(d, W, list(tokens), layers_out=trace).float()


def close(got, want, dev, what=""):
    """fp32: every value within 2e-4.  bf16: per row, the error (root mean square over the row) relative to the row's
    own spread is below 4 % on average and 40 % at the worst row."""
    diff = got.float().cpu() - want
    if dev[1] == torch.float32:
        err = diff.abs().max().item()
        assert err < 2e-4 * max(1.0, want.abs().max().item()), f"{what}: max abs error {err}"
        return
    rel = diff.pow(2).mean(-1).sqrt() / want.std(-1).clamp_min(1e-3)
    assert rel.mean().item() < 0.04 and rel.max().item() < 0.4, f"{what}: relative rms error mean {rel.mean()} max {rel.max()}"


def toks(n, vocab=50, seed=1):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def all_rows(n):
    return [list(range(n))]


def op_tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)


# ---- each mechanism alone, inside a one- or two-layer model ----------------------------------------------------
CASES = {
    "attention": cfg_dict([att(ff=0)]),
    "attention_unstretched": cfg_dict([att(scaling=None)]),
    "attention_every_entry_rotated": cfg_dict([att(rot=10)]),
    "attention_one_head": cfg_dict([att(heads=1, kv=1, dim=2, vdim=1, rot=2)]),
    "attention_a_key_head_per_query_head": cfg_dict([att(heads=5, kv=5)]),
    "attention_one_key_head": cfg_dict([att(heads=7, kv=1, vdim=12)]),
    "stretch_of_one": cfg_dict([att(scaling=yarn(factor=1.0)), lat(scaling=yarn(factor=1.0))]),
    "stretch_without_a_ramp": cfg_dict([att(scaling=yarn(fast=3.0, slow=3.0)), lat(scaling=yarn(original=6, fast=1.0, slow=1.0))]),
    "stretch_of_every_pair": cfg_dict([att(scaling=yarn(original=3, fast=100.0, slow=50.0, factor=16.0))]),
    "stretch_of_no_pair": cfg_dict([att(scaling=yarn(original=10 ** 9, fast=2.0, slow=1.0))]),
    "latent": cfg_dict([lat(ff=0)]),
    "latent_unstretched": cfg_dict([lat(scaling=None)]),
    "latent_one_head": cfg_dict([lat(heads=1, dim=3, rot=2, vdim=1, kv=5, qr=3)]),
    "recurrence": cfg_dict([ssm(ff=0)]),
    "recurrence_one_of_everything": cfg_dict([ssm(heads=1, vdim=1, state=1, groups=1, conv=1, parts=1)]),
    "recurrence_one_tap": cfg_dict([ssm(conv=1)]),
    "recurrence_two_taps": cfg_dict([ssm(conv=2)]),
    "recurrence_five_taps": cfg_dict([ssm(conv=5)]),
    "recurrence_a_group_per_head": cfg_dict([ssm(heads=5, groups=5, parts=5)]),
    "recurrence_a_norm_part_per_channel": cfg_dict([ssm(heads=2, vdim=3, parts=6)]),
    "weights_used_three_times": cfg_dict([ssm(), same_as(0, ssm()), att(), same_as(0, ssm())]),
    "weights_of_a_later_layer": cfg_dict([same_as(1, att()), att()]),
    "scales_of_one": cfg_dict([att(scale=1.0), lat(scale=1.0)], scale=1.0),
}


@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("case", list(CASES))
def test_each_mechanism_alone(dev, case):
    m = build(CASES[case], dev)
    t = toks(21, seed=4)
    want = oracle_logits(CASES[case], m, t)
    r = HybridRunner(m, 32)
    got = [r.step([("a", t[:13])], all_rows(13))]
    got += [r.step([("a", [x])]) for x in t[13:]]
    close(torch.cat(got), want, dev, case)


def test_traits_and_state_of_the_architecture():
    m = build(FULL, ("cpu", torch.float32))
    c = m.config
    assert (c.block, c.norm, c.dense_act, c.tied_head, c.embed_scale) == ("sandwich", "rms", "geglu", False, 3.0)
    assert c.latent == {"rot": "pairs", "gate": False, "sink": True, "p32": True}
    assert (c.attention["qk_norm"], c.attention["rot"], c.attention["gate"], c.attention["sink"]) == ("none", "halves", "head", False)
    assert m.blocks[4] is m.blocks[1] and m.blocks[8] is m.blocks[1] and m.blocks[5] is m.blocks[0] and m.blocks[7] is m.blocks[3]
    names = m.tensor_map()
    assert not any(n.startswith(("l4.", "l5.", "l6.", "l7.", "l8.")) for n in names)
    assert "l3.norm2" not in names and "l3.norm1b" in names and "l0.norm1.b" not in names and names["l2.mix.sink"].shape == (3,)
    pool = m.new_pool(3, 16)
    own = [t.data_ptr() for run in pool.runs for t in run.values()]
    assert len(set(own)) == len(own)  # shared weights, never a shared cache or state
    assert pool.runs[5]["state"].shape == (3, 4, 9, 6) and pool.runs[5]["state"].dtype == torch.float32
    assert pool.runs[5]["conv"].shape == (3, 3, 24 + 36) and pool.runs[4]["cache"].shape == (3, 16, 51)


@pytest.mark.parametrize("where", WHERE)
def test_shared_weights_equal_copied_weights(where):
    base = [att(), ssm()]
    shared = cfg_dict(base + [same_as(1, base[1]), same_as(0, base[0])])
    copied = cfg_dict(base + [base[1], base[0]])
    W = O.random_tensors(shared)
    both = dict(W)
    for n, v in W.items():
        for i, j in ((2, 1), (3, 0)):
            if n.startswith(f"l{j}."):
                both[f"l{i}." + n.split(".", 1)[1]] = v
    t = toks(19)
    a = HybridLM(HybridConfig.from_dict(shared)).load_tensors(W, where, torch.float32)
    b = HybridLM(HybridConfig.from_dict(copied)).load_tensors(both, where, torch.float32)
    ra, rb = HybridRunner(a, 32), HybridRunner(b, 32)
    for cut in (slice(0, 11), slice(11, 12), slice(12, 19)):
        torch.testing.assert_close(ra.step([("a", t[cut])]), rb.step([("a", t[cut])]), rtol=0, atol=0)


# ---- mechanisms as operations --------------------------------------------------------------------------------
@pytest.mark.parametrize("rot", [{"dims": 8, "base": 100.0}, {"dims": 16, "base": 10000.0, "scaling": yarn(8.0, 4096, 32.0, 1.0)},
                                 {"dims": 6, "base": 50.0, "scaling": yarn(3.0, 40, 2.0, 2.0)},
                                 {"dims": 12, "base": 7.0, "scaling": yarn(5.0, 10 ** 6, 1.0, 0.001)},
                                 {"dims": 2, "base": 3.0, "scaling": yarn(1.0, 5, 9.0, 0.1)}], ids=str)
def test_frequencies_and_amplitude(rot):
    got = H.scaled_inv_freq(rot["dims"], rot["base"], rot.get("scaling"), torch.device("cpu"))
    torch.testing.assert_close(got.double(), torch.tensor(O.frequencies(rot), dtype=torch.float64), rtol=1e-6, atol=0)
    assert H.rotary_amplitude(rot.get("scaling")) == pytest.approx(O.amplitude(rot), rel=1e-12)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("pairing", ["pairs", "halves"])
@pytest.mark.parametrize("nrot", [0, 2, 6, 10])
def test_preparation_of_grouped_heads(where, pairing, nrot):
    """Rotation only, in either pairing, of the first entries; queries in place, keys and values into the slot's rows."""
    Hh, G, D, V = 4, 2, 10, 3
    rot = {"dims": nrot, "base": 40.0, "scaling": yarn(6.0, 100, 6.0, 0.5)}
    g = torch.Generator().manual_seed(nrot)
    p = torch.randn(5, Hh * D + G * (D + V), generator=g)
    inv = H.scaled_inv_freq(nrot, 40.0, rot["scaling"], torch.device(where)) if nrot else None
    plan = BatchPlan.make([3, 2], [2, 0], [0, 71], torch.device(where))
    cache = torch.full((3, 80, G * (D + V)), 9.0, device=where)
    pw = p.clone().to(where)
    q, k, v = pw[:, :Hh * D], pw[:, Hh * D:Hh * D + G * D], pw[:, Hh * D + G * D:]
    H.window_append(q, k, v, inv, cache, plan, Hh, G, D, V, nrot, 1e-3, norm=False, pairing=pairing, amp=H.rotary_amplitude(rot["scaling"]))
    for row, (slot, pos) in enumerate([(2, 0), (2, 1), (2, 2), (0, 71), (0, 72)]):
        z = p[row].double()
        tv = [O.turn(z[a * D:(a + 1) * D], pos, rot, pairing == "pairs") if nrot else z[a * D:(a + 1) * D] for a in range(Hh + G)]
        torch.testing.assert_close(q[row].cpu().double(), torch.cat(tv[:Hh]), rtol=1e-5, atol=2e-5)
        torch.testing.assert_close(cache[slot, pos, :G * D].cpu().double(), torch.cat(tv[Hh:]), rtol=1e-5, atol=2e-5)
        torch.testing.assert_close(cache[slot, pos, G * D:].cpu(), p[row, Hh * D + G * D:], rtol=0, atol=0)
    assert (cache[1] == 9.0).all() and (cache[2, 3:] == 9.0).all() and (cache[0, :71] == 9.0).all()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("pairing", ["pairs", "halves"])
def test_preparation_of_the_latent_row(where, pairing):
    Q, L, R = 11, 14, 8
    rot = {"dims": 8, "base": 50.0, "scaling": yarn(4.0, 60, 4.0, 0.5)}
    g = torch.Generator().manual_seed(3)
    p, qw, w = torch.randn(5, Q + L + R, generator=g), torch.randn(Q, generator=g), torch.randn(L, generator=g)
    inv, amp = H.scaled_inv_freq(8, 50.0, rot["scaling"], torch.device(where)), H.rotary_amplitude(rot["scaling"])
    plan = BatchPlan.make([3, 2], [2, 0], [0, 7], torch.device(where))
    cache = torch.full((3, 12, L + R), 9.0, device=where)
    pw = p.to(where)
    cq = H.latent_prepare(pw[:, :Q], qw.to(where), pw[:, Q:], w.to(where), inv, cache, plan, R, L, 8, 1e-3, pairing, amp)
    heads = torch.randn(5, 3 * (4 + R), generator=g)
    turned = H.rotate_heads(heads.clone().to(where), inv, plan, 3, 4, R, 8, pairing, amp)
    for row, (slot, pos) in enumerate([(2, 0), (2, 1), (2, 2), (0, 7), (0, 8)]):
        z = p[row].double()
        torch.testing.assert_close(cq[row].cpu().double(), O.rms(z[:Q], qw.double(), 1e-3), rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(cache[slot, pos, :L].cpu().double(), O.rms(z[Q:Q + L], w.double(), 1e-3), rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(cache[slot, pos, L:].cpu().double(), O.turn(z[Q + L:], pos, rot, pairing == "pairs"), rtol=1e-5, atol=1e-5)
        for a in range(3):
            x = heads[row].double()[a * (4 + R):(a + 1) * (4 + R)]
            want = torch.cat((x[:4], O.turn(x[4:], pos, rot, pairing == "pairs")))
            torch.testing.assert_close(turned[row].cpu().double()[a * (4 + R):(a + 1) * (4 + R)], want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(9, 4), (64, 4), (64, 1), (136, 2), (1032, 3), (24, 5)])
def test_convolution_in_steps_of_every_size(where, dtype, C, taps):
    """Three packed sequences in scattered slots; steps of one token, of fewer tokens than taps, of many, in any order."""
    g = torch.Generator().manual_seed(C + taps)
    w, b = torch.randn(C, taps, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype)
    xs = {s: torch.randn(70, C, generator=g).to(dtype) for s in (4, 0, 2)}
    want = {}
    for s, x in xs.items():
        past, rows = [], []
        for row in x.double():
            past.append(row)
            rows.append(O.silu(O.short_conv(w.double(), b.double(), past)))
        want[s] = torch.stack(rows).float()
    state = torch.zeros(5, max(0, taps - 1), C, dtype=dtype)
    state[1], state[3] = 77.0, 77.0
    state = state.to(where)
    at = {s: 0 for s in xs}
    for sizes in ((1, 2, 7), (1, 1, 1), (2, 1, 4), (40, 1, 1), (1, 17, 2), (1, 1, 1), (3, 2, 50)):
        plan = BatchPlan.make(sizes, list(xs), [at[s] for s in xs], torch.device(where))
        x = torch.cat([xs[s][at[s]:at[s] + n] for s, n in zip(xs, sizes)])
        wide = torch.full((x.size(0), C + 16), 5.0, dtype=dtype)
        wide[:, 8:8 + C] = x
        got = H.conv_silu(wide.to(where)[:, 8:8 + C], w.to(where), state, plan, b.to(where))
        row = 0
        for s, n in zip(xs, sizes):
            torch.testing.assert_close(got[row:row + n].float().cpu(), want[s][at[s]:at[s] + n], **op_tol(dtype))
            row, at[s] = row + n, at[s] + n
    if taps > 1:
        assert (state[1] == 77.0).all() and (state[3] == 77.0).all()


def _ssd_case(dtype, Hh, G, N, V, lengths, seed, dt_mean, a_mean):
    g = torch.Generator().manual_seed(seed)
    T = sum(lengths)
    xbc = torch.randn(T, Hh * V + 2 * G * N, generator=g).to(dtype)
    xbc[:, Hh * V:] *= 0.7
    dt = (dt_mean + torch.randn(T, Hh, generator=g)).to(dtype)
    return xbc, dt, 0.3 * torch.randn(Hh, generator=g), a_mean + 0.5 * torch.randn(Hh, generator=g), torch.randn(Hh, generator=g)


def _plain_ssd(xbc, dt, bias, a_log, d, S, Hh, G, N, V):
    out = []
    x_, B, C = (t.double() for t in xbc.float().split((Hh * V, G * N, G * N), 1))
    S = [s for s in S.double()]
    for t in range(xbc.size(0)):
        ys = []
        for a in range(Hh):
            gi = a // (Hh // G)
            S[a], y = O.state_step(S[a], x_[t, a * V:(a + 1) * V], B[t, gi * N:(gi + 1) * N], C[t, gi * N:(gi + 1) * N],
                                   O.softplus(dt[t, a].double() + bias[a].double()), a_log[a].double(), d[a].double())
            ys.append(y)
        out.append(torch.cat(ys))
    return torch.stack(out).float(), torch.stack(S).float()


SSD_SHAPES = [(2, 1, 5, 3), (4, 2, 16, 16), (3, 3, 24, 40), (2, 2, 128, 64), (2, 1, 64, 136), (1, 1, 1, 1), (1, 1, 200, 8)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SSD_SHAPES, ids=str)
@pytest.mark.parametrize("speed", ["slow", "mixed", "fast"])
def test_state_space_recurrence_in_every_form(where, dtype, shape, speed):
    """Unequal sequences in scattered slots, the first with a state from before; the token scan and the chunked form.
    ``fast``: the decay of a few tokens underflows; ``slow``: a chunk hardly decays at all."""
    Hh, G, N, V = shape
    dt_mean, a_mean = {"slow": (-3.0, -3.0), "mixed": (-1.0, 0.0), "fast": (3.0, 4.0)}[speed]
    lengths, slots = [291, 1, 64, 17], [3, 0, 2, 4]
    xbc, dt, bias, a_log, d = _ssd_case(dtype, Hh, G, N, V, lengths, 5, dt_mean, a_mean)
    start = torch.zeros(6, Hh, N, V)
    start[3] = torch.randn(Hh, N, V, generator=torch.Generator().manual_seed(8))
    start[1], start[5] = 1e3, 1e3
    want, finals, r0 = [], [], 0
    for n, s in zip(lengths, slots):
        y, S = _plain_ssd(xbc[r0:r0 + n], dt[r0:r0 + n], bias, a_log, d, start[s], Hh, G, N, V)
        want.append(y), finals.append(S)
        r0 += n
    want = torch.cat(want)
    plan = BatchPlan.make(lengths, slots, [9, 0, 0, 0], torch.device(where))
    wide = torch.cat((xbc.new_zeros(xbc.size(0), 8), dt, xbc.new_zeros(xbc.size(0), 5)), 1).to(where)
    forms = [0] if where == "cpu" else ([0, 1, 2] if dtype == torch.bfloat16 else [0, 1])
    for variant in forms:
        state = start.clone().to(where)
        plan.shared.clear()
        got = H.ssd_recurrence(xbc.to(where), wide[:, 8:8 + Hh], bias.to(where), a_log.to(where), d.to(where), state, plan, Hh, G, N, V,
                               variant)
        scale = max(1.0, want.abs().max().item())
        torch.testing.assert_close(got.cpu(), want, rtol=1e-4, atol=5e-5 * scale)  # whatever the activation type: the state is fp32
        torch.testing.assert_close(state[slots].cpu(), torch.stack(finals), rtol=1e-4, atol=5e-5 * max(1.0, start[3].abs().max().item(), scale))
        assert (state[1] == 1e3).all() and (state[5] == 1e3).all()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("at", [0, 1, 15, 16, 62, 63, 64, 65, 126, 127, 128, 199])
def test_one_loud_token_is_remembered_across_chunks(where, at):
    """All inputs are nearly silent but one token's; with a slow decay every later read-out is that token's, none earlier."""
    Hh, N, V, T = 2, 16, 16, 200
    dtype = torch.bfloat16 if where == "cuda" else torch.float32
    g = torch.Generator().manual_seed(at)
    xbc = 1e-3 * torch.randn(T, Hh * V + 2 * N, generator=g)
    xbc[:, Hh * V + N:] = torch.randn(T, N, generator=g)
    xbc[at, :Hh * V + N] = 5.0 * torch.randn(Hh * V + N, generator=g)
    xbc, dt = xbc.to(dtype), torch.full((T, Hh), -2.0, dtype=dtype)
    bias, a_log, d = torch.zeros(Hh), torch.full((Hh,), -3.0), torch.zeros(Hh)
    want, _ = _plain_ssd(xbc, dt, bias, a_log, d, torch.zeros(Hh, N, V), Hh, 1, N, V)
    assert want[at:].abs().amax(1).min() > 100 * (want[:at].abs().max() if at else 0.0)
    for cuts in ((T,), (at + 1, T - at - 1), (70, 2, T - 72)):
        state, got, p0 = torch.zeros(1, Hh, N, V, device=where), [], 0
        for n in (c for c in cuts if c):
            plan = BatchPlan.make([n], [0], [p0], torch.device(where))
            got.append(H.ssd_recurrence(xbc[p0:p0 + n].to(where), dt[p0:p0 + n].to(where), bias.to(where), a_log.to(where), d.to(where), state,
                                        plan, Hh, 1, N, V))
            p0 += n
        torch.testing.assert_close(torch.cat(got).cpu(), want, rtol=1e-3, atol=1e-3)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,parts", [(12, 1), (12, 4), (9, 9), (64, 2), (4096, 1), (4096, 8), (5000, 5), (9000, 1)])
def test_gate_then_norm_in_parts(where, dtype, n, parts):
    g = torch.Generator().manual_seed(n + parts)
    y, w = 3.0 * torch.randn(4, n, generator=g), (1 + 0.2 * torch.randn(n, generator=g)).to(dtype)
    y[:, :n // parts] *= 50.0  # the parts' sizes differ: a norm over the whole row would show
    y[2] = 0.0
    wide = torch.randn(4, n + 24, generator=g).to(dtype)
    want = torch.stack([O.gate_and_norm(y[i].double(), wide[i, 8:8 + n].double(), w.double(), parts, 1e-5) for i in range(4)]).float()
    got = H.silu_gate_norm(y.to(where), wide.to(where)[:, 8:8 + n], w.to(where), parts, 1e-5, dtype)
    assert got.dtype == dtype
    torch.testing.assert_close(got.float().cpu(), want, **op_tol(dtype))


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [13, 64])
def test_gated_feed_forward(where, dtype, ff):
    m = GatedFF(20, ff, "gelu_tanh")
    g = torch.Generator().manual_seed(ff)
    for p in (m.gate, m.up, m.down):
        p.data = (2.0 * torch.randn(p.shape, generator=g) * p.shape[1] ** -0.5).to(where, dtype)
    m.finalize()
    h = torch.randn(6, 20, generator=g).to(where, dtype)
    W = {n: getattr(m, n).double().cpu() for n in ("gate", "up", "down")}
    want = torch.stack([O.feed_forward(W, "", r) for r in h.double().cpu()]).float()
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    torch.testing.assert_close(m(h).float().cpu(), want, **tol)


# ---- both attentions: a key that stands out, forms against each other -----------------------------------------
def _latent(where, dtype, Hh, D, R, V, L, scale=1.0):
    m = LatentAttention(32, {"heads": Hh, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": L, "q_rank": 8, "scale": scale,
                             "rot": {"dims": R, "base": 100.0, "scaling": yarn(2.0, 64, 8.0, 1.0)}}, 1e-6,
                        {"rot": "pairs", "gate": False, "sink": True, "p32": True})
    g = torch.Generator().manual_seed(Hh + L)
    for name, p in m.named_parameters():
        p.data = (torch.randn(p.shape, generator=g) * p.shape[-1] ** -0.5).to(where, dtype)
    m.sink.data = (1.0 + torch.randn(Hh, generator=g)).to(where, dtype)
    m.finalize()
    return m, {"dims": R, "base": 100.0, "scaling": yarn(2.0, 64, 8.0, 1.0)}


def _plain_latent(m, rot, q, cache, pos):
    """One query row ``[H * (D + R)]`` (not rotated) at ``pos`` over cache rows ``[positions, L + R]``; float64."""
    D, R, V, L = m.D, m.R, m.V, m.L
    rows, outs = cache[:pos + 1].double().cpu(), []
    for a in range(m.H):
        qa = q.double().cpu()[a * (D + R):(a + 1) * (D + R)]
        k = rows[:, :L] @ m.uk.double().cpu()[a * D:(a + 1) * D].T
        v = rows[:, :L] @ m.uv.double().cpu()[a * V:(a + 1) * V].T
        s = (k @ qa[:D] + rows[:, L:] @ O.turn(qa[D:], pos, rot, True)) * m.scale
        outs.append(O.softmax_sum(s, v, m.sink.double().cpu()[a]))
    return torch.stack(outs)


LAT_SHAPES = [(3, 6, 4, 5, 10), (4, 16, 16, 24, 32), (2, 32, 16, 80, 128), (17, 8, 8, 16, 96), (16, 48, 16, 128, 512)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LAT_SHAPES[:3], ids=str)
@pytest.mark.parametrize("sink", [-40.0, 0.0, 6.0, 33.0])
def test_latent_attention_far_key_and_sink(where, dtype, shape, sink):
    """Head 0 has one key that takes nearly all the weight unless the sink does: at the start, at tile edges, at the token
    itself, just after it (left in the slot by an earlier user).  One-token form with any number of key shares, prompt form."""
    Hh, D, R, V, L = shape
    m, rot = _latent(where, dtype, Hh, D, R, V, L, scale=(D + R) ** -0.5)
    m.sink.data[0] = sink
    m.finalize()
    g = torch.Generator().manual_seed(7)
    S, pos, dev = 256, 201, torch.device(where)
    q = torch.randn(1, Hh * (D + R), generator=g).to(where, dtype)
    qr = O.turn(q[0].double().cpu()[D:D + R], pos, rot, True)
    loud = (30.0 / m.scale * qr / (qr @ qr)).to(dtype)
    for at in (0, 1, 31, 32, 64, 127, 128, pos, pos + 1):
        cache = torch.zeros(3, S, L + R)
        cache[1] = 0.5 * torch.randn(S, L + R, generator=g)
        cache[1, at, L:] = loud.float()
        cache = cache.to(where, dtype)
        want = _plain_latent(m, rot, q[0], cache[1], pos)
        if at <= pos and sink <= 6.0:
            alone = m.uv.double().cpu().view(Hh, V, L)[0] @ cache[1, at, :L].double().cpu()
            assert (want[0] - alone).abs().max() < 0.05  # nothing else than this key
        if sink == 33.0:
            assert want[0].abs().max() < 0.3             # and here hardly even this one
        plan = BatchPlan.make([1], [1], [pos], dev)
        qlat = H.matmul_f32(q.view(1, Hh, D + R)[:, :, :D].transpose(0, 1), m.uk.view(Hh, D, L))
        tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
        for split in ((0, 1, 2, 5, 32) if where == "cuda" else (0,)):
            olat = H.latent_attn(qlat, q, cache, plan, Hh, D, R, L, m.scale, split=split, inv_freq=m.inv_freq, nrot=R, pairing="pairs",
                                 amp=m.amp, sink=m.sink32)
            got = torch.einsum("hl,hvl->hv", olat[:, 0].double().cpu(), m.uv.double().cpu().view(Hh, V, L))
            torch.testing.assert_close(got.float(), want.float(), **tol)
        for n, band, fused in ((70, 17, False), (pos + 1, 64, False), (64, 64, True), (79, 64, True), (pos + 1, 64, True)):
            m.query_block, m.fused_prompt = band, fused  # the query is the last row of a portion of n tokens
            qs = torch.randn(n, Hh * (D + R), generator=g).to(where, dtype)
            qs[-1] = q[0]
            plan = BatchPlan.make([n], [1], [pos + 1 - n], dev)
            H.rotate_heads(qs, m.inv_freq, plan, Hh, D, R, R, "pairs", m.amp)
            torch.testing.assert_close(m._expanded(qs, cache, plan)[-1].float().cpu(), want.float(), **tol)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LAT_SHAPES, ids=str)
def test_latent_attention_on_unequal_sequences_in_scattered_slots(where, dtype, shape):
    Hh, D, R, V, L = shape
    m, rot = _latent(where, dtype, Hh, D, R, V, L, scale=(D + R) ** -0.5)
    g = torch.Generator().manual_seed(11)
    cache = torch.randn(4, 160, L + R, generator=g).to(where, dtype)
    lengths, slots, starts = [70, 1, 3, 66], [2, 0, 3, 1], [0, 0, 0, 90]
    plan = BatchPlan.make(lengths, slots, starts, torch.device(where))
    N = sum(lengths)
    q = torch.randn(N, Hh * (D + R), generator=g).to(where, dtype)
    rows = [r0 + i for (r0, n, _, _) in plan.seqs for i in range(0, n, 1 if n < 5 else 13)]
    want = {r0 + i: _plain_latent(m, rot, q[r0 + i], cache[slot], p0 + i) for (r0, n, slot, p0) in plan.seqs for i in range(n) if r0 + i in rows}
    want = torch.stack([want[r] for r in rows]).float()
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    qlat = H.matmul_f32(q.view(N, Hh, D + R)[:, :, :D].transpose(0, 1), m.uk.view(Hh, D, L))
    olat = H.latent_attn(qlat, q, cache, plan, Hh, D, R, L, m.scale, inv_freq=m.inv_freq, nrot=R, pairing="pairs", amp=m.amp, sink=m.sink32)
    got = torch.einsum("hnl,hvl->nhv", olat.double().cpu(), m.uv.double().cpu().view(Hh, V, L))
    torch.testing.assert_close(got[rows].float(), want, **tol)
    H.rotate_heads(q, m.inv_freq, plan, Hh, D, R, R, "pairs", m.amp)
    for m.fused_prompt in (True, False):
        torch.testing.assert_close(m._expanded(q, cache, plan)[rows].float().cpu(), want, **tol)


def _grouped(where, dtype, Hh, G, D, V, scale, window=0, sink=None):
    mixer = {"heads": Hh, "kv_heads": G, "dim": D, "vdim": V, "scale": scale}
    if window:
        mixer["mask"] = {"size": window}
    m = WindowAttention(24, mixer, 1e-6, {"qk_norm": "none", "rot": "halves", "gate": "head", "p32": True, "sink": "learned" if sink else False})
    g = torch.Generator().manual_seed(Hh * D)
    for name, p in m.named_parameters():
        p.data = (torch.randn(p.shape, generator=g) * p.shape[-1] ** -0.5).to(where, dtype)
    if sink:
        m.sink_w.data = torch.full((Hh,), sink).to(where, dtype)
    m.finalize()
    return m


def _plain_grouped(m, q, gate, cache, pos):
    Hh, G, D, V = m.H, m.G, m.D, m.V
    lo = max(0, pos - m.window + 1) if m.window else 0
    rows, outs = cache[lo:pos + 1].double().cpu(), []
    for a in range(Hh):
        b = a // (Hh // G)
        s = rows[:, b * D:(b + 1) * D] @ q.double().cpu()[a * D:(a + 1) * D] * m.scale
        sk = m.sink_w.double().cpu()[a] if m.sink_w is not None else None
        outs.append(O.softmax_sum(s, rows[:, G * D + b * V:G * D + (b + 1) * V], sk) * O.sigmoid(gate.double().cpu()[a]))
    return torch.cat(outs)


GQA_SHAPES = [(4, 2, 10, 7), (6, 3, 32, 16), (20, 1, 64, 48), (5, 5, 16, 128), (9, 3, 128, 64), (2, 1, 48, 256)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", GQA_SHAPES, ids=str)
@pytest.mark.parametrize("window,sink", [(0, None), (0, 2.0), (50, None), (64, 1.0)])
def test_grouped_attention_forms_on_unequal_sequences(where, dtype, shape, window, sink):
    """The per-token form, the fused prompt kernel and the banded matrix products, on the same cache; a key that stands out
    for the last row of each sequence sits at the first visible position, one before it, at tile edges, at the token itself and after it."""
    Hh, G, D, V = shape
    m = _grouped(where, dtype, Hh, G, D, V, D ** -0.5, window, sink)
    g = torch.Generator().manual_seed(13)
    lengths, slots, starts = [130, 64, 67], [2, 0, 3], [0, 0, 75]
    plan = BatchPlan.make(lengths, slots, starts, torch.device(where))
    N = sum(lengths)
    q, gate = torch.randn(N, Hh * D, generator=g).to(where, dtype), torch.randn(N, Hh, generator=g).to(where, dtype)
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    for case in range(7):
        cache = torch.randn(4, 160, G * (D + V), generator=g)
        for (r0, n, slot, p0) in plan.seqs:
            last = p0 + n - 1
            lo = max(0, last - window + 1) if window else 0
            at = [lo, max(0, lo - 1), last, last + 1, 31, 32, 63][case]
            qa = q[r0 + n - 1].float().cpu().view(Hh, D)[0]
            cache[slot, at, :D] = 25.0 * qa / (qa @ qa) * D ** 0.5
        cache = cache.to(where, dtype)
        rows = [r0 + i for (r0, n, _, _) in plan.seqs for i in ({n - 1} if case else {0, 1, 30, 63, n - 1})]
        where_of = {r0 + i: (slot, p0 + i) for (r0, n, slot, p0) in plan.seqs for i in range(n)}
        want = torch.stack([_plain_grouped(m, q[r], gate[r], cache[where_of[r][0]], where_of[r][1]) for r in rows]).float()
        for split, mma in (((0, True), (1, True), (2, True), (7, True), (32, True), (0, False), (5, False)) if where == "cuda" else ((0, True),)):
            got = H.window_attn(q, gate, cache, plan, Hh, G, D, V, m.scale, window, split, sink=sink is not None, sink_vals=m.sink32, mma=mma)
            torch.testing.assert_close(got[rows].float().cpu(), want, **tol)
        got = H.head_gate(m._banded(q, cache, plan), gate)
        torch.testing.assert_close(got[rows].float().cpu(), want, **tol)
        if m._takes_fused(q):
            plan.shared.clear()
            torch.testing.assert_close(m._fused(q, gate, cache, plan)[rows].float().cpu(), want, **tol)
    if where == "cuda":
        assert m._takes_fused(q) == (dtype == torch.bfloat16 and shape != GQA_SHAPES[0])


@pytest.mark.gpu
@pytest.mark.parametrize("mask,window,sink,cap,gate", [("chunk", 48, True, 0.0, "channel"), ("window", 0, "learned", 15.0, "head"),
                                                       ("chunk", 64, "learned", 0.0, None), ("window", 20, False, 5.0, "channel")])
def test_single_token_attention_variants_agree_with_the_fp32_form(mask, window, sink, cap, gate):
    """The tensor-core form and the form on fp32 values, on one-token steps of unequal contexts with every mask, sink, gate and cap."""
    Hh, G, D, V = 6, 2, 32, 48
    g = torch.Generator().manual_seed(3)
    starts = [0, 1, 15, 16, 47, 48, 63, 64, 127, 150]
    n = len(starts)
    plan = BatchPlan.make([1] * n, list(range(n)), starts, torch.device("cuda"))
    bf = dict(device="cuda", dtype=torch.bfloat16)
    q, cache = torch.randn(n, Hh * D, generator=g).to(**bf), torch.randn(n, 160, G * (D + V), generator=g).to(**bf)
    gt = None if gate is None else torch.randn(n, Hh * (V if gate == "channel" else 1), generator=g).to(**bf)
    sv = torch.randn(Hh, generator=g).cuda() if sink == "learned" else None
    kw = dict(mask=mask, sink=bool(sink), cap=cap, sink_vals=sv)
    for split in (0, 1, 3):
        a = H.window_attn(q, gt, cache, plan, Hh, G, D, V, 0.3, window, split, **kw)
        b = H.window_attn(q, gt, cache, plan, Hh, G, D, V, 0.3, window, split, mma=False, **kw)
        torch.testing.assert_close(a.float(), b.float(), rtol=1e-2, atol=1e-2)


# ---- whole models: prompts, decoding, portions, batches, slots ------------------------------------------------
@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("d", [FULL, FULL32], ids=["odd", "aligned"])
def test_whole_prompts_and_first_tokens(dev, d, monkeypatch):
    monkeypatch.setattr(LatentAttention, "query_block", 48)  # a prompt runs in several bands of query rows
    monkeypatch.setattr(WindowAttention, "query_block", 48)
    m = build(d, dev)
    for n in (1, 2, 3, 4, 15, 16, 17, 63, 64, 65, 129, 150):
        t = toks(n, seed=n)
        close(HybridRunner(m, 160).step([("a", t)], all_rows(n)), oracle_logits(d, m, t), dev, f"prompt of {n}")


@pytest.mark.parametrize("dev", DEVICES)
def test_residual_trace(dev):
    m = build(FULL, dev)
    t = toks(9)
    want = []
    oracle_logits(FULL, m, t, want)
    pool = m.new_pool(1, 16)
    plan = BatchPlan.make([len(t)], [pool.alloc()], [0], m.device)
    got = []
    m(torch.tensor(t, dtype=torch.int32, device=m.device), plan, pool, trace=got)
    assert len(got) == want[0].shape[0] == 9
    for i, x in enumerate(got):
        close(x, want[0][i].float(), dev, f"stream after layer {i}")


@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("d", [FULL, FULL32], ids=["odd", "aligned"])
def test_prefill_then_long_decode(dev, d):
    m = build(d, dev)
    t = toks(170, seed=3)
    want = oracle_logits(d, m, t)
    r = HybridRunner(m, 192)
    got = [r.step([("a", t[:30])], all_rows(30))]
    for p in range(30, 170):
        got.append(r.step([("a", [t[p]])]))
    close(torch.cat(got), want, dev, "decode")
    r2 = HybridRunner(m, 128)
    one = torch.cat([r2.step([("b", [x])]) for x in t[:20]])
    close(one, want[:20], dev, "token by token")


@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("cuts", [(2, 3, 2, 64, 5, 70, 1, 2, 11), (66, 2, 92), (15, 1, 16, 40, 41, 63, 2), (180,)],
                         ids=["small", "mixed", "edges", "whole"])
def test_portions_of_a_prompt(dev, cuts):
    d = FULL32 if cuts[0] in (66, 15) else FULL
    m = build(d, dev)
    t = toks(sum(cuts), seed=5)
    want = oracle_logits(d, m, t)
    r = HybridRunner(m, 288)
    got, at = [], 0
    for c in cuts:
        got.append(r.step([("a", t[at:at + c])], all_rows(c)))
        at += c
    close(torch.cat(got), want, dev, f"portions {cuts}")


@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("d", [FULL, FULL32], ids=["odd", "aligned"])
@pytest.mark.parametrize("lengths", [(5, 19, 1, 9), (75, 64, 141), (80, 1, 3)], ids=["short", "long", "mixed"])
def test_unequal_batch_equals_each_alone_and_slots_are_reused(dev, d, lengths):
    m = build(d, dev)
    seqs = {f"s{i}": toks(n + 12, seed=10 + i) for i, n in enumerate(lengths)}
    want = {k: oracle_logits(d, m, v) for k, v in seqs.items()}
    r = HybridRunner(m, 192, n_slots=2)  # the pool has to grow
    live = list(seqs)
    out = r.step([(k, seqs[k][:n]) for k, n in zip(live, lengths)], [list(range(n)) for n in lengths])
    at = 0
    for k, n in zip(live, lengths):
        close(out[at:at + n], want[k][:n], dev, f"prompt {k}")
        at += n
    pos = dict(zip(live, lengths))
    rows, refs = [], []
    for stepno in range(12):
        if stepno == 4:  # one request ends early; its slot goes back
            r.end_sample(live.pop(1))
        out = r.step([(k, [seqs[k][pos[k]]]) for k in live])
        for i, k in enumerate(live):
            rows.append(out[i:i + 1])
            refs.append(want[k][pos[k]:pos[k] + 1])
            pos[k] += 1
    close(torch.cat(rows), torch.cat(refs), dev, "batched decode")
    for k in live:
        r.end_sample(k)
    assert not r.pool.length
    t = toks(75, seed=99)  # freed slots serve a new request: nothing of the old cache, convolution inputs or state shows
    w = oracle_logits(d, m, t)
    close(r.step([("new", t[:1])]), w[:1], dev, "reused slot, first token")
    close(r.step([("new", t[1:3])], all_rows(2)), w[1:3], dev, "reused slot, next two")
    close(r.step([("new", t[3:])], all_rows(72)), w[3:], dev, "reused slot, rest")


@pytest.mark.parametrize("dev", DEVICES)
def test_pool_grows_while_requests_are_held(dev):
    m = build(FULL32, dev)
    seqs = [toks(n, seed=40 + i) for i, n in enumerate((80, 66, 140, 71, 5))]
    want = [oracle_logits(FULL32, m, t) for t in seqs]
    r = HybridRunner(m, 192, n_slots=2)
    r.step([(0, seqs[0][:70]), (1, seqs[1][:60])])
    rows, refs = [], []

    def advance(s):
        out = r.step([(0, [seqs[0][70 + s]]), (1, [seqs[1][60 + s]])])
        rows.append(out)
        refs.append(torch.stack((want[0][70 + s], want[1][60 + s])))

    for s in range(3):  # the third one-token step of this batch size runs as a captured graph on the GPU
        advance(s)
    out = r.step([(i, seqs[i]) for i in (2, 3, 4)])
    assert r.pool.n_slots >= 5
    rows.append(out)
    refs.append(torch.stack([want[i][-1] for i in (2, 3, 4)]))
    for s in range(3, 6):
        advance(s)
    close(torch.cat(rows), torch.cat(refs), dev, "before and after growth")


@pytest.mark.parametrize("dev", DEVICES)
def test_greedy_generation_through_the_runner(dev):
    m = build(FULL, dev)
    prompts = [toks(5, seed=1), toks(11, seed=2)]
    r = HybridRunner(m, 32)
    out = r.generate(prompts, 6, SamplingParams.greedy())
    assert not r.pool.length and [len(o) for o in out] == [11, 17]
    if dev[1] == torch.float32:
        for p, o in zip(prompts, out):
            seq = list(p)
            for _ in range(6):
                seq.append(int(oracle_logits(FULL, m, seq)[-1].argmax()))
            assert o == seq


# ---- checkpoint, registry, command line ---------------------------------------------------------------------
def _save(m, ck):
    ck.mkdir()
    m.config.save(ck)
    tensors = {k: v.to(torch.bfloat16) for k, v in m.state_tensors().items()}
    write_safetensors(tensors, ck / "model.safetensors")
    return tensors


def test_checkpoint_roundtrip_registry_and_trace_cli(tmp_path):
    m = build(FULL, ("cpu", torch.float32))
    ck = tmp_path / "ck"
    tensors = _save(m, ck)
    cfg_cls, model_cls = model_classes("Dufelix")
    assert cfg_cls is HybridConfig and model_cls is HybridLM
    m2 = load_hybrid(ck, "cpu", torch.float32)
    c = m2.config
    assert HybridConfig.from_dict(c.asdict()).asdict() == c.asdict() and c.layers[8]["weights_of"] == 1 and c.norm_eps == 1e-3
    for gone in ("l2.mix.sink", "l0.mix.conv.b", "head", "l1.mlp.gate", "l2.mix.dkv.norm", "l3.mix.A_log", "l0.norm2b"):
        with pytest.raises(KeyError):
            HybridLM(c).load_tensors({k: v for k, v in tensors.items() if k != gone}, "cpu", torch.float32)
    with pytest.raises(KeyError):  # a layer with another layer's weights has none
        HybridLM(c).load_tensors({**tensors, "l4.mix.q": tensors["l1.mix.q"]}, "cpu", torch.float32)
    t = toks(12)
    want = oracle_logits(FULL, m2, t)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:8], "want": [0, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[8:9], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[9:10], "want": [0]}, ], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": t, "want": [11]}], "end": ["y"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(ck), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "16", "--device", "cpu"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    import numpy as np

    def rd(i):
        return torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, 50).copy())

    assert not (out / "1.f32").exists()
    for i, rows in ((0, [0, 7]), (2, [9]), (3, [11])):
        close(rd(i), want[rows], ("cpu", torch.float32))


def test_sample_command_line_serves_the_checkpoint(tmp_path, capsys):
    from mdi_llm_b200.cli import sample

    m = build(FULL32, ("cpu", torch.float32))
    _save(m, tmp_path / "ck")
    assert sample.main(["--ckpt", str(tmp_path / "ck"), "--prompt", "two cats", "--n-samples", "2", "--n-tokens", "5", "--greedy",
                        "--device", "cpu", "--dtype", "float32"]) == 0
    out = capsys.readouterr().out
    ids = [b % 50 for b in b"two cats"]
    want = []
    for _ in range(5):
        want.append(int(oracle_logits(FULL32, m, ids + want)[-1].argmax()))
    assert out.count(" ".join(map(str, want))) == 2, out


def test_config_validation():
    bad = [cfg_dict([same_as(1, att()), same_as(0, att())]),        # nobody has the tensors
           cfg_dict([att(), same_as(2, att())]), cfg_dict([att(), same_as(0, att(heads=3))]),
           cfg_dict([ssm(heads=5)]), cfg_dict([ssm(parts=5)]), cfg_dict([ssm(conv=0)]), cfg_dict([att(kv=4)]),
           dict(cfg_dict([att(), same_as(0, att())]), token_side={"dim": 4})]
    for d in bad:
        with pytest.raises(ValueError):
            HybridConfig.from_dict(d)
    chain = HybridConfig.from_dict(cfg_dict([att(), same_as(0, att()), same_as(1, att())]))
    assert [chain.weights_layer(i) for i in range(3)] == [0, 0, 0]
    with pytest.raises(ValueError):
        HybridLM(HybridConfig.from_dict(cfg_dict([att(rot=12)])))
    m = build(FULL, ("cpu", torch.float32))
    with pytest.raises(ValueError):
        HybridRunner(m, 8).step([("a", toks(9))])
    assert math.isclose(H.rotary_amplitude(yarn(1.0)), 1.0) and H.rotary_amplitude(None) == 1.0
