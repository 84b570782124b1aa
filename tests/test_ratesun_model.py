"""The Ratesun design (sandwich blocks with input convolutions and an average over depth, windowed latent attention on
shared caches) against the plain oracle of ``ratesun_oracle.py``.

Every test builds its own small configuration with random weights.  Sizes are awkward on purpose: value width != key
width, widths that are not a multiple of four beside some that are, windows of one token up to longer than the sequence,
a layer that borrows another layer's cache with a window, heads and value width of its own, one to five convolution
taps, a layer without feed-forward, one bucket in the bigram table.  The same tests run on the CPU (PyTorch bodies of
the operations) and, marked ``gpu``, on the sm_100a kernels.
"""
from __future__ import annotations

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import ratesun_oracle as O
from mdi_llm_b200.models.config import HybridConfig
from mdi_llm_b200.models.hybrid import HybridLM, LatentAttention, load_hybrid, write_safetensors
from mdi_llm_b200.models.registry import model_classes
from mdi_llm_b200.ops import hybrid as H
from mdi_llm_b200.ops.hybrid import BatchPlan
from mdi_llm_b200.parallel.hybrid_runner import HybridRunner
from mdi_llm_b200.parallel.scheduler import SamplingParams

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def layer(heads=3, dim=10, rot=6, vdim=7, kv=14, qr=11, scale=0.3, size=9, base=500.0, kv_from=None, ff=20, rot_dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv, "q_rank": qr, "scale": scale,
         "rot": {"dims": rot if rot_dims is None else rot_dims, "base": base}}
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def cfg_dict(layers, width=22, vocab=50, eps=1e-3, taps=3, side=5, mult=0.6, scale=1.7, bigram=(37, 11, 5)):
    d = {"architecture": "Ratesun", "vocab": vocab, "width": width, "layers": copy.deepcopy(layers), "norm": {"eps": eps},
         "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "canon": {"taps": taps},
         "residual_mult": mult, "logit_scale": scale}
    if side:
        d["token_side"] = {"dim": side}
    return d


# an own cache, a borrower with other heads, value width and a wider window, a layer with 16-byte rows and its borrower
# with a window of one, a layer without feed-forward; and the same with a width in whole 16-byte groups
LAYERS = [layer(), layer(heads=5, dim=4, vdim=9, qr=6, scale=0.7, size=40, kv_from=0, ff=24),
          layer(heads=2, dim=16, rot=8, vdim=16, kv=32, qr=16, scale=0.2, size=70, base=10000.0, ff=16),
          layer(heads=4, dim=8, rot=8, vdim=24, kv=32, qr=24, scale=1.1, size=1, base=10000.0, kv_from=2, ff=0),
          layer(heads=1, size=33, ff=12)]
FULL = cfg_dict(LAYERS)
FULL32 = cfg_dict(LAYERS[:4], width=32, taps=4, side=8, eps=1e-6)

DEVICES = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
           pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]
WHERE = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]


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
    own spread is below 8 % on average and 40 % at the worst row."""
    diff = got.float().cpu() - want
    if dev[1] == torch.float32:
        err = diff.abs().max().item()
        assert err < 2e-4 * max(1.0, want.abs().max().item()), f"{what}: max abs error {err}"
        return
    rel = diff.pow(2).mean(-1).sqrt() / want.std(-1).clamp_min(1e-3)
    assert rel.mean().item() < 0.08 and rel.max().item() < 0.4, f"{what}: relative rms error mean {rel.mean()} max {rel.max()}"


def toks(n, vocab=50, seed=1):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def all_rows(n):
    return [list(range(n))]


# ---- each mechanism alone, inside a one- or two-layer model ----------------------------------------------------
CASES = {
    "window": cfg_dict([layer(ff=0)], taps=1, side=0),
    "window_of_one": cfg_dict([layer(size=1, ff=0)]),
    "window_longer_than_the_sequence": cfg_dict([layer(size=500)]),
    "no_window": cfg_dict([layer(size=0)]),
    "one_head": cfg_dict([layer(heads=1, dim=3, rot=2, vdim=1, kv=5, qr=3)]),
    "part_of_the_key_part_rotated": cfg_dict([layer(rot=8, rot_dims=4)]),
    "borrowed_cache": cfg_dict([layer(), layer(heads=7, dim=5, vdim=3, qr=4, scale=0.9, size=3, kv_from=0)]),
    "one_tap": cfg_dict([layer()], taps=1),
    "two_taps": cfg_dict([layer()], taps=2),
    "five_taps": cfg_dict([layer()], taps=5, width=24),
    "no_side": cfg_dict([layer(), layer(kv_from=0)], side=0),
    "multipliers_of_one": cfg_dict([layer(scale=1.0)], mult=1.0, scale=1.0),
    "one_bucket": cfg_dict([layer()], bigram=(1, 3, 2)),
    "large_multipliers": cfg_dict([layer()], bigram=(41, 2_000_000_011, 1_999_999_973)),
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
    assert (c.block, c.norm, c.dense_act, c.depth_average, c.tied_head) == ("sandwich", "layer", "polynorm", True, True)
    assert c.latent == {"rot": "pairs", "gate": False, "sink": False, "p32": True}
    pool = m.new_pool(3, 16)
    assert pool.runs[1]["cache"] is pool.runs[0]["cache"] and pool.runs[3]["cache"] is pool.runs[2]["cache"]
    assert pool.runs[0]["canon1"].shape == (3, 2, 22) and pool.runs[0]["canon1"].dtype == torch.float32
    assert "canon2" not in pool.runs[3] and pool.prev.shape == (3,)
    names = m.tensor_map()
    assert "l1.mix.dkv" not in names and "l1.mix.dkv.norm" not in names and "l1.mix.uk" in names
    assert names["l4.dwa"].shape == (6,) and names["bigram"].shape == (38, 22) and "l3.norm2" not in names


# ---- mechanisms as operations --------------------------------------------------------------------------------
DTYPES = [torch.float32, torch.bfloat16]


def op_tol(dtype):
    return dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("F", [1, 20, 256, 1000, 4096, 16384, 20000])
def test_polynomial_activation(where, dtype, F):
    z = torch.randn(5, F, generator=torch.Generator().manual_seed(F)).to(dtype)
    z[1] *= 30.0
    z[2] = 0.0
    coef = torch.tensor([0.8, -0.3, 0.6, 0.2])
    want = torch.stack([O.poly_norm(r.double(), coef.double(), 1e-4) for r in z.float()]).float()
    got = H.poly_norm(z.to(where), coef.to(where), 1e-4)
    torch.testing.assert_close(got.float().cpu(), want, **op_tol(dtype))


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("C", [6, 24])
def test_bigram_rows_follow_the_previous_token_of_the_slot(where, C):
    buckets, mp, mc = 23, 7, 13
    table, pair = torch.randn(30, C), torch.randn(buckets + 1, C)
    prev = torch.full((4,), 29, dtype=torch.int32, device=where)  # what earlier users of the slots left
    seqs = {2: [3, 0, 29, 7], 0: [5], 3: [1, 1, 2]}
    at = {s: 0 for s in seqs}

    def step(brings):
        slots = list(brings)
        plan = BatchPlan.make([brings[s] for s in slots], slots, [at[s] for s in slots], torch.device(where))
        tk = [seqs[s][at[s] + i] for s in slots for i in range(brings[s])]
        out2 = torch.empty(len(tk), C, device=where)
        out = H.embed_pairs(table.to(where), pair.to(where), torch.tensor(tk, dtype=torch.int32, device=where), plan, prev, buckets, mp, mc,
                            1.5, out2=out2)
        assert torch.equal(out, out2)
        row = 0
        for s in slots:
            for _ in range(brings[s]):
                p, t = at[s], seqs[s][at[s]]
                b = buckets if p == 0 else (seqs[s][p - 1] * mp + t * mc) % buckets
                torch.testing.assert_close(out[row].cpu(), 1.5 * table[t] + pair[b])
                row, at[s] = row + 1, at[s] + 1

    step({2: 1, 0: 1, 3: 2})
    step({3: 1, 2: 1})
    step({2: 2})
    assert prev.tolist()[2] == 7 and prev.tolist()[0] == 5 and prev.tolist()[1] == 29


def _plain_norm_conv(x, w, b, eps, conv, taps):
    past, out = [], []
    for row in x.double():
        past.append(O.layer_norm(row, w.double(), b.double(), eps))
        out.append(O.short_conv(conv.double(), past))
    return torch.stack(out).float()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(10, 3), (64, 4), (64, 1), (132, 2), (1028, 5)])
@pytest.mark.parametrize("tile", [0, 1, 3, 16])
def test_norm_and_convolution_in_steps_of_every_size(where, dtype, C, taps, tile):
    """Three packed sequences in scattered slots whose state holds another user's rows; steps of one token, of fewer tokens
    than taps, of many, in any order: every row is what the whole sequence gives."""
    g = torch.Generator().manual_seed(C + taps)
    w, b, conv = (1 + 0.2 * torch.randn(C, generator=g)).to(dtype), (0.2 * torch.randn(C, generator=g)).to(dtype), torch.randn(C, taps, generator=g)
    xs = {4: 3 * torch.randn(29, C, generator=g) + 1, 0: torch.randn(29, C, generator=g), 2: torch.randn(29, C, generator=g)}
    want = {s: _plain_norm_conv(x, w.float(), b.float(), 1e-5, conv, taps) for s, x in xs.items()}
    state = torch.full((5, max(0, taps - 1), C), 1e4, device=where)
    nxt = H.NextInput(w.to(where), b.to(where), 1e-5, "layer", conv.t().contiguous().to(where), state)
    at = {s: 0 for s in xs}
    for sizes in ((1, 2, 7), (1, 1, 1), (2, 1, 4), (9, 1, 1), (1, 17, 2), (1, 1, 1), (3, 2, 1)):
        plan = BatchPlan.make(sizes, list(xs), [at[s] for s in xs], torch.device(where))
        x = torch.cat([xs[s][at[s]:at[s] + n] for s, n in zip(xs, sizes)]).to(where)
        got = H.norm_conv(x, nxt, plan, dtype, tile)
        row = 0
        for s, n in zip(xs, sizes):
            torch.testing.assert_close(got[row:row + n].float().cpu(), want[s][at[s]:at[s] + n], **op_tol(dtype))
            row, at[s] = row + n, at[s] + n
    if taps > 1:
        assert (state[1] == 1e4).all() and (state[3] == 1e4).all()  # nobody's slots are not touched


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C", [9, 64, 1300])
@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_residual_update_with_depth_average_and_next_input(where, dtype, C, kind):
    g = torch.Generator().manual_seed(C)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    N, index, taps = 3, 4, 3
    depth, y, w, b = r(7, N, C), (2 * r(N, C) + 0.5).to(dtype), (1 + 0.2 * r(C)).to(dtype), (0.3 * r(C)).to(dtype)
    w2, b2, conv, dw, old = (1 + 0.2 * r(C)).to(dtype), (0.3 * r(C)).to(dtype), r(C, taps), r(index + 1), r(N, taps - 1, C)
    bias = b if kind == "layer" else None
    want_x, want_avg, want_h = [], [], []
    starts = [5, 0, 1]  # the second sequence has no past, the third one row of it: what else the slot holds counts as zero
    for i in range(N):
        yd = y[i].double()
        n = O.layer_norm(yd, w.double(), b.double(), 1e-4) if kind == "layer" else O.rms(yd, w.double(), 1e-4)
        x = depth[index, i].double() + 0.7 * n
        avg = O.depth_average(dw.double(), [depth[j, i].double() for j in range(index)] + [x])
        past = list(old[i].double())[max(0, taps - 1 - starts[i]):] + [O.layer_norm(avg, w2.double(), b2.double(), 1e-4)]
        want_x.append(x), want_avg.append(avg), want_h.append((O.short_conv(conv.double(), past), past[-1]))
    d, state = depth.to(where), torch.full((4, taps - 1, C), 1e3, device=where)
    slots = [3, 0, 2]
    for i, s in enumerate(slots):
        state[s] = old[i].to(where)
    plan = BatchPlan.make([1] * N, slots, starts, torch.device(where))
    nxt = H.NextInput(w2.to(where), b2.to(where), 1e-4, "layer", conv.t().contiguous().to(where), state)
    copy_ = torch.empty(N, C, dtype=dtype, device=where)
    h = H.row_update(d[index], y.to(where), w.to(where), None if bias is None else bias.to(where), 1e-4, kind, 0.7, copy=copy_, depth=d,
                     index=index, depth_w=dw.to(where), nxt=nxt, plan=plan, out_dtype=dtype)
    torch.testing.assert_close(d[index].cpu(), torch.stack(want_x).float(), rtol=2e-5, atol=2e-5)
    torch.testing.assert_close(copy_.float().cpu(), torch.stack(want_x).float(), **op_tol(dtype))
    torch.testing.assert_close(d[index + 1].cpu(), torch.stack(want_avg).float(), rtol=2e-5, atol=5e-5)
    torch.testing.assert_close(h.float().cpu(), torch.stack([a for a, _ in want_h]).float(), **(op_tol(dtype) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)))
    torch.testing.assert_close(state[slots, -1].cpu(), torch.stack([s for _, s in want_h]).float(), rtol=1e-4, atol=1e-4)
    assert torch.equal(d[:index].cpu(), depth[:index]) and torch.equal(d[index + 2:].cpu(), depth[index + 2:])
    assert (state[1] == 1e3).all()
    # without a sublayer output only the average is taken; without an average only the update
    d2 = depth.to(where)
    H.row_update(d2[index], depth=d2, index=index, depth_w=dw.to(where))
    torch.testing.assert_close(d2[index + 1].cpu(), torch.einsum("j,jnc->nc", dw, depth[:index + 1]), rtol=1e-4, atol=1e-4)


def _attention(where, dtype, Hh, D, R, V, L, W, base=100.0, scale=1.0):
    m = LatentAttention(32, {"heads": Hh, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": L, "q_rank": 8, "scale": scale,
                             "rot": {"dims": R, "base": base}, "mask": {"size": W}}, 1e-6, {"rot": "pairs", "gate": False, "p32": True})
    g = torch.Generator().manual_seed(W + L)
    for name, p in m.named_parameters():
        p.data = (torch.randn(p.shape, generator=g) * p.shape[-1] ** -0.5).to(where, dtype)
    m.finalize()
    return m


def _plain_attention(m, q, cache, pos):
    """One query row ``[H * (D + R)]`` (not rotated) at ``pos`` over cache rows ``[positions, L + R]``; float64."""
    D, R, V, L, W = m.D, m.R, m.V, m.L, m.window
    first = max(0, pos - W + 1) if W else 0
    rows = cache[first:pos + 1].double().cpu()
    outs = []
    for a in range(m.H):
        qa = q.double().cpu()[a * (D + R):(a + 1) * (D + R)]
        k = rows[:, :L] @ m.uk.double().cpu()[a * D:(a + 1) * D].T
        v = rows[:, :L] @ m.uv.double().cpu()[a * V:(a + 1) * V].T
        s = (k @ qa[:D] + rows[:, L:] @ O.turn_pairs(qa[D:], pos, R, m.rot_base)) * m.scale
        outs.append(O.softmax(s) @ v)
    return torch.stack(outs)


SHAPES = [(3, 6, 4, 5, 10), (4, 16, 16, 24, 32), (2, 32, 16, 80, 128), (17, 8, 8, 16, 96), (16, 48, 16, 128, 512)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [1, 16, 33, 64, 150])
@pytest.mark.parametrize("shape", SHAPES[:3], ids=str)
def test_one_key_stands_out_just_inside_and_outside_the_window_and_later(where, dtype, W, shape):
    """A key that takes nearly all the weight at the window's first position, one before it, at the token itself, one after
    it (left in the slot by an earlier user), and in the middle: one-token form with any number of key shares, and the
    prompt form with its bands starting at several places."""
    Hh, D, R, V, L = shape
    m = _attention(where, dtype, Hh, D, R, V, L, W)
    g = torch.Generator().manual_seed(7)
    S, pos = 256, 201
    dev = torch.device(where)
    q = torch.randn(1, Hh * (D + R), generator=g).to(where, dtype)
    # the rotated key part that answers head 0's rotated query part: its score is far above the others'
    qr = O.turn_pairs(q[0].double().cpu()[D:D + R], pos, R, m.rot_base)
    loud = (30.0 * qr / (qr @ qr)).to(dtype)
    for at in sorted({pos - W, pos - W + 1, pos - W // 2, pos, pos + 1, 0}):
        cache = torch.zeros(3, S, L + R)
        cache[1] = 0.5 * torch.randn(S, L + R, generator=g)
        cache[1, at, L:] = loud.float()
        cache = cache.to(where, dtype)
        want = _plain_attention(m, q[0], cache[1], pos)
        visible = pos - W < at <= pos
        assert (want - (m.uv.double().cpu().view(Hh, V, L) @ cache[1, at, :L].double().cpu())).abs()[0].max() < 0.02 or not visible
        plan = BatchPlan.make([1], [1], [pos], dev)
        qlat = H.matmul_f32(q.view(1, Hh, D + R)[:, :, :D].transpose(0, 1), m.uk.view(Hh, D, L))
        tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
        for split in ((0, 1, 2, 5, 32) if where == "cuda" else (0,)):
            olat = H.latent_attn(qlat, q, cache, plan, Hh, D, R, L, m.scale, split=split, window=W, inv_freq=m.inv_freq, nrot=R, pairing="pairs")
            got = torch.einsum("hl,hvl->hv", olat[:, 0].double().cpu(), m.uv.double().cpu().view(Hh, V, L))
            torch.testing.assert_close(got.float(), want.float(), **tol)
        for n, band, fused in ((64, 1024, False), (70, 17, False), (pos + 1, 64, False), (64, 64, True), (79, 64, True), (pos + 1, 64, True)):
            m.query_block, m.fused_prompt = band, fused  # the query is the last row of a portion of n tokens
            qs = torch.randn(n, Hh * (D + R), generator=g).to(where, dtype)
            qs[-1] = q[0]
            plan = BatchPlan.make([n], [1], [pos + 1 - n], dev)
            H.rotate_heads(qs, m.inv_freq, plan, Hh, D, R, R, "pairs")
            torch.testing.assert_close(m._expanded(qs, cache, plan)[-1].float().cpu(), want.float(), **tol)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("W", [0, 50])
def test_both_forms_on_unequal_sequences_in_scattered_slots(where, dtype, shape, W):
    Hh, D, R, V, L = shape
    m = _attention(where, dtype, Hh, D, R, V, L, W, scale=(D + R) ** -0.5)
    g = torch.Generator().manual_seed(11)
    cache = torch.randn(4, 160, L + R, generator=g).to(where, dtype)
    lengths, slots, starts = [70, 1, 3, 66], [2, 0, 3, 1], [0, 0, 0, 90]
    plan = BatchPlan.make(lengths, slots, starts, torch.device(where))
    N = sum(lengths)
    q = torch.randn(N, Hh * (D + R), generator=g).to(where, dtype)
    want = torch.empty(N, Hh, V)
    for (r0, n, slot, p0) in plan.seqs:
        for i in range(0, n, 1 if n < 5 else 13):
            want[r0 + i] = _plain_attention(m, q[r0 + i], cache[slot], p0 + i)
    rows = [r0 + i for (r0, n, _, _) in plan.seqs for i in range(0, n, 1 if n < 5 else 13)]
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    qlat = H.matmul_f32(q.view(N, Hh, D + R)[:, :, :D].transpose(0, 1), m.uk.view(Hh, D, L))
    olat = H.latent_attn(qlat, q, cache, plan, Hh, D, R, L, m.scale, window=W, inv_freq=m.inv_freq, nrot=R, pairing="pairs")
    got = torch.einsum("hnl,hvl->nhv", olat.double().cpu(), m.uv.double().cpu().view(Hh, V, L))
    torch.testing.assert_close(got[rows].float(), want[rows], **tol)
    H.rotate_heads(q, m.inv_freq, plan, Hh, D, R, R, "pairs")
    for m.fused_prompt in (True, False):
        torch.testing.assert_close(m._expanded(q, cache, plan)[rows].float().cpu(), want[rows], **tol)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("pairing", ["pairs", "halves"])
def test_preparation_norms_rotates_and_writes_the_cache_row(where, pairing):
    Q, L, R, nrot = 11, 14, 8, 6
    g = torch.Generator().manual_seed(3)
    p, qw, w = torch.randn(5, Q + L + R, generator=g), torch.randn(Q, generator=g), torch.randn(L, generator=g)
    inv = H.rotary_inv_freq(nrot, 50.0, torch.device(where))
    plan = BatchPlan.make([3, 2], [2, 0], [0, 7], torch.device(where))
    cache = torch.full((3, 12, L + R), 9.0, device=where)
    pw = p.to(where)
    cq = H.latent_prepare(pw[:, :Q], qw.to(where), pw[:, Q:], w.to(where), inv, cache, plan, R, L, nrot, 1e-3, pairing)
    for row, (slot, pos) in enumerate([(2, 0), (2, 1), (2, 2), (0, 7), (0, 8)]):
        z = p[row].double()
        torch.testing.assert_close(cq[row].cpu().double(), O.rms(z[:Q], qw.double(), 1e-3), rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(cache[slot, pos, :L].cpu().double(), O.rms(z[Q:Q + L], w.double(), 1e-3), rtol=1e-5, atol=1e-5)
        k = z[Q + L:]
        if pairing == "halves":
            order = [0, 3, 1, 4, 2, 5, 6, 7]  # (i, i + nrot/2) become neighbours
            t = O.turn_pairs(k[order], pos, nrot, 50.0)
            kk = torch.empty_like(t)
            kk[order] = t
        else:
            kk = O.turn_pairs(k, pos, nrot, 50.0)
        torch.testing.assert_close(cache[slot, pos, L:].cpu().double(), kk, rtol=1e-5, atol=1e-5)
    before = cache.clone()
    cq2 = H.latent_prepare(pw[:, :Q], qw.to(where), None, None, inv, cache, plan, R, L, nrot, 1e-3, pairing)  # a borrower
    assert torch.equal(cq, cq2) and torch.equal(cache, before) and (cache[1] == 9.0).all()


# ---- whole models: prompts, decoding, portions, batches, slots ------------------------------------------------
@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("d", [FULL, FULL32], ids=["odd", "aligned"])
def test_whole_prompts_and_first_tokens(dev, d, monkeypatch):
    monkeypatch.setattr(LatentAttention, "query_block", 48)  # a prompt runs in several bands of query rows
    m = build(d, dev)
    for n in (1, 2, 3, 9, 10, 40, 41, 63, 64, 65, 71, 150):  # the first tokens; just inside and outside every window
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
    assert len(got) == want[0].shape[0] == 5
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
    for p in range(30, 170):  # every window passes over prompt tokens, then over decoded ones
        got.append(r.step([("a", [t[p]])]))
    close(torch.cat(got), want, dev, "decode")
    r2 = HybridRunner(m, 128)
    one = torch.cat([r2.step([("b", [x])]) for x in t[:20]])
    close(one, want[:20], dev, "token by token")


@pytest.mark.parametrize("dev", DEVICES)
@pytest.mark.parametrize("cuts", [(2, 3, 2, 64, 5, 70, 1, 2, 11), (66, 2, 92), (9, 1, 10, 40, 41, 69, 2), (230,)],
                         ids=["small", "mixed", "window_edges", "whole"])
def test_portions_of_a_prompt(dev, cuts):
    d = FULL32 if cuts[0] == 66 else FULL
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
@pytest.mark.parametrize("lengths", [(5, 19, 1, 9), (75, 64, 141), (80, 1, 3)], ids=["short", "long", "mixed"])
def test_unequal_batch_equals_each_alone_and_slots_are_reused(dev, lengths):
    d = FULL
    m = build(d, dev)
    seqs = {f"s{i}": toks(n + 12, seed=10 + i) for i, n in enumerate(lengths)}
    want = {k: oracle_logits(d, m, v) for k, v in seqs.items()}
    r = HybridRunner(m, 192, n_slots=2)  # the pool has to grow; borrowed caches must follow
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
    t = toks(75, seed=99)  # freed slots serve a new request: nothing of the old cache, convolutions or last token shows
    w = oracle_logits(d, m, t)
    close(r.step([("new", t[:1])]), w[:1], dev, "reused slot, first token")
    close(r.step([("new", t[1:3])], all_rows(2)), w[1:3], dev, "reused slot, next two")
    close(r.step([("new", t[3:])], all_rows(72)), w[3:], dev, "reused slot, rest")
    for run, (li, _) in zip(r.pool.runs, m.config.layer_runs()):  # a borrowed cache is the lender's tensor, also after growth
        src = m.config.layers[li]["mixer"].get("kv_from")
        if src is not None:
            assert run["cache"] is r.pool.runs[src]["cache"]


@pytest.mark.parametrize("dev", DEVICES)
def test_pool_grows_while_requests_are_held(dev):
    m = build(FULL, dev)
    seqs = [toks(n, seed=20 + i) for i, n in enumerate((80, 66, 140, 71, 5))]
    want = [oracle_logits(FULL, m, t) for t in seqs]
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
    cfg_cls, model_cls = model_classes("Ratesun")
    assert cfg_cls is HybridConfig and model_cls is HybridLM
    m2 = load_hybrid(ck, "cpu", torch.float32)
    c = m2.config
    assert HybridConfig.from_dict(c.asdict()).asdict() == c.asdict()
    assert c.canon_taps == 3 and c.bigram == {"buckets": 37, "mul_prev": 11, "mul_cur": 5} and c.logit_scale == 1.7
    for gone in ("l2.dwa", "l0.canon2", "bigram", "l1.mlp.act", "l2.mix.dkv.norm"):
        with pytest.raises(KeyError):
            HybridLM(c).load_tensors({k: v for k, v in tensors.items() if k != gone}, "cpu", torch.float32)
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
    assert sample.main(["--ckpt", str(tmp_path / "ck"), "--prompt", "rate of suns", "--n-samples", "2", "--n-tokens", "5", "--greedy",
                        "--device", "cpu", "--dtype", "float32"]) == 0
    out = capsys.readouterr().out
    ids = [b % 50 for b in b"rate of suns"]
    want = []
    for _ in range(5):
        want.append(int(oracle_logits(FULL32, m, ids + want)[-1].argmax()))
    assert out.count(" ".join(map(str, want))) == 2, out


def test_config_validation():
    bad = [cfg_dict([layer(kv_from=1), layer()]),                      # the lender comes first
           cfg_dict([layer(), layer(kv_from=0), layer(kv_from=1)]),    # and has a cache of its own
           cfg_dict([layer(), layer(kv=16, kv_from=0)]),               # whose rows the borrower understands
           cfg_dict([layer(), layer(base=501.0, kv_from=0)]),
           cfg_dict([layer()], bigram=(0, 1, 1)), cfg_dict([layer()], taps=-1),
           dict(cfg_dict([layer(), layer()]), loop={"start": 0, "stop": 1, "times": 2}),
           dict(cfg_dict([layer()]), architecture="Vudelix")]          # input convolutions belong to sandwich blocks
    for d in bad:
        with pytest.raises(ValueError):
            HybridConfig.from_dict(d)
    with pytest.raises(ValueError):
        HybridLM(HybridConfig.from_dict(cfg_dict([layer(rot=6, rot_dims=5)])))
    m = build(FULL, ("cpu", torch.float32))
    with pytest.raises(ValueError):
        HybridRunner(m, 8).step([("a", toks(9))])
