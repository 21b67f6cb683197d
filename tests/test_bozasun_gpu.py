"""The Bozasun design on the device against the plain NumPy restatement (oracle/bozasun.py), in fp32 and bf16."""

import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import bozasun as OB
from oracle import fuzudra as OF
from oracle.fuzudra import bf16
import bozasun_cases as BC
from bozasun_cases import Expected, build, err, greedy, prompt
from test_fuzudra_cpu import write_model
from test_fuzudra_gpu import in_portions, whole

pytestmark = pytest.mark.gpu
DTYPES = ["f32", "bf16"]

A, L, M, E = BC.attention, BC.latent, BC.mamba, BC.moe
MECHANISMS = {
    "attention": A(), "attention_one_head": A(heads=1, kv_heads=1, dim=5, vdim=7, rot=4, chunk=2),
    "attention_all_rotated": A(dim=32, vdim=32, rot=32, chunk=64), "attention_unscaled_uncapped": A(factor=None, softcap=None, chunk=65),
    "attention_wide": A(heads=4, kv_heads=1, dim=128, vdim=96, rot=64, chunk=100, scale=0.1), "attention_no_chunks": A(chunk=None),
    "attention_many_heads_per_key": A(heads=20, kv_heads=1, dim=16, vdim=24, rot=8, chunk=50), "attention_narrow": A(heads=5, kv_heads=5, dim=8, vdim=4, rot=4),
    "attention_dim_180": A(heads=2, kv_heads=1, dim=180, vdim=64, rot=90, scale=0.08), "attention_vdim_250": A(heads=2, kv_heads=2, dim=40, vdim=250),
    "attention_dim_300": A(heads=1, kv_heads=1, dim=300, vdim=20, scale=0.06), "attention_low_cap": A(softcap=0.8, scale=1.5),
    "latent": L(), "latent_one_head": L(heads=1, dim=5, rot_dim=2, vdim=7, kv_rank=3), "latent_wide": L(heads=6, dim=64, rot_dim=32, vdim=48, kv_rank=160, scale=0.1),
    "latent_more_rotated": L(heads=2, dim=8, rot_dim=40, vdim=16, kv_rank=24, base=50.0), "latent_many_heads": L(heads=20, dim=16, rot_dim=8, vdim=16, kv_rank=100),
    "latent_rank_512": L(heads=2, dim=16, rot_dim=64, vdim=16, kv_rank=512, mlp=None), "latent_rank_270": L(heads=3, dim=32, rot_dim=48, vdim=16, kv_rank=270, mlp=None),
    "latent_rank_beyond_tiles": L(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=640, mlp=None),
    "mamba": M(), "mamba_one_head": M(heads=1, vdim=5, state=3, groups=1, norm_groups=1, conv=2), "mamba_state_128": M(heads=4, vdim=64, state=128, groups=1, norm_groups=1),
    "mamba_state_64": M(heads=3, vdim=72, state=64, groups=3, norm_groups=3), "mamba_state_160": M(heads=2, vdim=40, state=160, groups=2), "mamba_state_300": M(heads=2, vdim=12, state=300, groups=1),
    "mamba_vdim_150": M(heads=2, vdim=150, state=40, groups=1, norm_groups=2), "mamba_one_tap": M(conv=1), "mamba_six_taps": M(conv=6, heads=4, vdim=16, state=16, groups=4, norm_groups=8),
    "moe_plain": M(mlp=E(groups=1, keep=1, identity=0, experts=6, top=2)), "moe_identity_only_chosen": M(mlp=E(experts=1, identity=9, top=3, groups=5, keep=3)),
    "moe_one_chosen": M(mlp=E(top=1)), "moe_many": L(mlp=E(experts=40, identity=8, top=6, groups=6, keep=3, ff=40)), "moe_all": M(mlp=E(experts=4, identity=2, top=6, groups=2, keep=2, ff=9)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_alone(name, dtype):
    cfg = BC.config([MECHANISMS[name]])
    sd = BC.weights(cfg, seed=3)
    toks = prompt(cfg, 150, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [70, 1, 2, 1, 40, 1]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", BC.MODELS)
def test_models_whole_portions_and_decoding(name, dtype):
    cfg = BC.MODELS[name]
    sd = BC.weights(cfg, seed=5)
    toks = prompt(cfg, 170, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    res = m.residuals(toks)
    assert len(res) == len(want.runs)
    for i, (a, b, tol) in enumerate(zip(res, want.runs, want.run_tol)):
        assert err(a, b) < tol[dtype], i
    want.check(whole(m, toks), dtype)
    for sizes in ([2], [1], [3, 2, 61, 1, 5], [64], [63, 65], [127, 1, 1, 40], [100] + [1] * 70):
        want.check(in_portions(m, toks, sizes), dtype, what=sizes)


@pytest.mark.parametrize("part", ["mix.q.b", "mix.k.b", "mix.v.b", "mix.o.b", "mix.q.norm", "side.embed", "side.proj", "side.norm", "mlp.router", "mlp.e2.up"])
def test_single_parts_scaled_up(part):
    """One part of a layer made the dominant one, in turn: an error in it cannot hide behind the others."""
    cfg = BC.config([A(chunk=20, mlp=E(experts=5, identity=1, top=3, groups=2, keep=2)), A(chunk=12)])
    sd = BC.weights(cfg, seed=21)
    sd[part if part == "side.embed" else "l0." + part] = bf16(3 * sd[part if part == "side.embed" else "l0." + part])
    toks = prompt(cfg, 80, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, "f32")
    want.check(whole(m, toks), "f32")
    want.check(in_portions(m, toks, [30, 1, 1, 2]), "f32")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_correction_moves_choices_but_not_weights(dtype):
    """Corrections far larger than the scores: all groups but the corrected ones are out, negative choice scores stay in."""
    cfg = BC.config([M(mlp=E(experts=6, identity=2, top=3, groups=4, keep=2))])
    sd = BC.weights(cfg, seed=17)
    for shift in ([0, 0, -3, -3, 0, 0, -3, -3], [-2] * 4 + [-5] * 4, [0, 4, -9, -9, -9, -9, 4, 0]):
        sd["l0.mlp.correction"] = bf16(np.array(shift, np.float32))
        toks = prompt(cfg, 60, seed=3, sd=sd)
        want = Expected(sd, cfg, toks)
        m = build(cfg, sd, dtype)
        want.check(whole(m, toks), dtype, what=shift)
        want.check(in_portions(m, toks, [1, 40]), dtype, what=shift)


ASKS, ANSWERS, FILLER = 95, 96, 90


def asking_model(layer):
    """Attention in which token ASKS finds token ANSWERS and nothing else: the first half of an embedding is what a token
    asks for, the second half what it offers, and these two share one vector."""
    cfg = BC.config([layer], width=64)
    sd = BC.weights(cfg, seed=9)
    eye, off = np.eye(32, dtype=np.float32), np.zeros((32, 32), np.float32)
    sd["embed"][ANSWERS, 32:] = sd["embed"][ASKS, :32]
    sd["l0.norm1"] = np.ones(64, np.float32)
    ask, offer = np.concatenate([eye, off], 1), np.concatenate([off, eye], 1)
    for n in ("q", "k"):
        for t, v in ((".b", 0), (".norm", 1)):
            if f"l0.mix.{n}{t}" in sd:
                sd[f"l0.mix.{n}{t}"] = sd[f"l0.mix.{n}{t}"] * 0 + v
    if layer["type"] == "attention":
        sd["l0.mix.q"], sd["l0.mix.k"] = np.tile(ask, (2, 1)), offer
    else:
        r = layer["mixer"]["rot_dim"]
        sd["l0.mix.q"] = np.tile(np.concatenate([ask, np.zeros((r, 64), np.float32)]), (2, 1))
        sd["l0.mix.dkv"][:32] = offer
        sd["l0.mix.dkv.norm"] = np.ones(32, np.float32)
        sd["l0.mix.uk"] = np.tile(eye, (2, 1))
    sd["l0.mix.o"] = bf16(sd["l0.mix.o"] * 4)
    return cfg, sd


def edge_layer(chunk):
    return A(heads=2, kv_heads=1, dim=32, vdim=32, chunk=chunk, rot=2, scale=0.4, factor=None, softcap=20.0, mlp=None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [2, 15, 16, 17, 63, 64, 65, 100])
def test_chunk_edges(chunk, dtype):
    """The answer at the first token of the asking token's chunk and just before it: in a prompt, in a portion, and when the
    asking token is decoded alone; the asking token at the chunk's first, second and last place and in between."""
    cfg, sd = asking_model(edge_layer(chunk))
    m = build(cfg, sd, dtype)
    first = chunk * (1 + 70 // chunk)
    base = prompt(cfg, first + chunk + 1) % FILLER
    for q in sorted({first, first + 1, first + chunk // 2, first + chunk - 1}):
        logits = {}
        for at in (first, first - 1):
            toks = base[:q + 1].copy()
            toks[q] = ASKS
            if at < q:
                toks[at] = ANSWERS
            want = Expected(sd, cfg, toks)
            for got in (whole(m, toks)[-1:], in_portions(m, toks, [q, 1])[-1:], in_portions(m, toks, [q - 4, 5])[-1:]):
                want.check(got, dtype, slice(q, q + 1), (q, at))
            logits[at] = want.logits[-1:]
        if q > first + 1:      # the case means something: the answer weighs
            assert err(logits[first], logits[first - 1]) > 3 * want.tol["bf16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_far_keys_at_page_borders(kind, dtype):
    """The answer hundreds of tokens back, at the first token and around page borders, while the asking token is decoded;
    many key ranges are merged."""
    cfg, sd = asking_model(edge_layer(None) if kind == "attention" else
                           L(heads=2, dim=32, rot_dim=6, vdim=32, kv_rank=32, scale=0.4, mlp=None))
    m = build(cfg, sd, dtype)
    base = prompt(cfg, 700, seed=4) % FILLER
    plain = None
    for at in (None, 0, 1, 63, 64, 65, 511, 512, 640):
        toks = base.copy()
        toks[-1] = ASKS
        if at is not None:
            toks[at] = ANSWERS
        want = Expected(sd, cfg, toks)
        plain = want.logits[-1:] if at is None else plain
        assert at is None or err(want.logits[-1:], plain) > 2 * want.tol["bf16"]
        for got in (whole(m, toks)[-1:], in_portions(m, toks, [699, 1])[-1:], in_portions(m, toks, [300, 395, 5])[-1:]):
            want.check(got, dtype, slice(699, 700), at)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_carries_a_far_token(dtype):
    """Slow decay: the first token's share of the state is still there hundreds of tokens later, across portions, chunks and
    decoded tokens."""
    cfg = BC.config([M(heads=2, vdim=24, state=24, groups=1, norm_groups=1)], width=64)
    sd = BC.weights(cfg, seed=31)
    sd["l0.mix.A_log"] = bf16(np.array([-9.0, -7.0], np.float32))
    sd["l0.mix.dt_bias"] = bf16(np.array([0.5, 0.5], np.float32))
    sd["l0.mix.in"][-2:] = bf16(sd["l0.mix.in"][-2:] * 0.1)
    sd["embed"][7] *= 30                                             # after the norm a token of its own kind
    sd["l0.mix.o"] = bf16(sd["l0.mix.o"] * 4)
    toks = prompt(cfg, 500, seed=2) % 90 + 8
    last = {}
    for first in (7, 8):
        t = toks.copy()
        t[0] = first
        want = Expected(sd, cfg, t)
        last[first] = want.logits[-1:]
        m = build(cfg, sd, dtype)
        want.check(whole(m, t)[-1:], dtype, slice(499, 500))
        want.check(in_portions(m, t, [64, 1, 63, 2, 150, 200, 1])[-1:], dtype, slice(499, 500))
    assert err(last[7], last[8]) > 3e-4                              # ten times what fp32 is allowed


def test_fast_and_slow_decays_in_one_chunk():
    """Steps that wipe the state out beside steps that leave it alone: exponents of a chunk far apart."""
    cfg = BC.config([M(heads=4, vdim=16, state=16, groups=2, norm_groups=1)], width=64)
    sd = BC.weights(cfg, seed=33)
    sd["l0.mix.A_log"] = bf16(np.array([4.0, -6.0, 2.0, 0.0], np.float32))
    sd["l0.mix.in"][-4:] = bf16(sd["l0.mix.in"][-4:] * 4)
    toks = prompt(cfg, 200, seed=2)
    want = Expected(sd, cfg, toks)
    for dtype in DTYPES:
        m = build(cfg, sd, dtype)
        want.check(whole(m, toks), dtype)
        want.check(in_portions(m, toks, [90, 1, 64, 2]), dtype)


@functools.lru_cache(None)
def wide_case():
    cfg = BC.config([M(heads=4, vdim=64, state=64, groups=2, norm_groups=2, mlp=E(experts=6, identity=2, top=3, groups=4, keep=3, ff=192)),
                     A(heads=8, kv_heads=2, dim=64, vdim=64, rot=64, chunk=150, scale=0.15, mlp=BC.dense(384)),
                     L(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, scale=0.1, mlp=E(experts=4, identity=4, top=2, groups=2, keep=1, ff=128)),
                     M(heads=2, vdim=128, state=128, groups=1, norm_groups=1, mlp=None)], width=256, vocab=300, side=32)
    sd = BC.weights(cfg, seed=6)
    toks = prompt(cfg, 540, sd=sd)
    return cfg, sd, toks, Expected(sd, cfg, toks)


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_layers_and_long_prompts(dtype):
    """Widths at which the bf16 model takes the many-row tensor-core route, a prompt over several row and state segments and
    several pieces of an expert's rows, and more rows of decoding than one key page."""
    cfg, sd, toks, want = wide_case()
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [460] + [1] * 80), dtype)
    want.check(in_portions(m, toks, [300, 7, 233]), dtype)
    want.check(in_portions(m, toks, [258, 282]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["plain", "other_order"])
def test_batches_slots_and_pages_are_used_again(name, dtype):
    """Unequal requests that come and go over a pool that holds only a part of them: every position equals the request
    alone; portions beside single tokens; requests that pause; a slot used by a longer request before."""
    import versenext_b200 as vn
    cfg = BC.MODELS[name]
    sd = BC.weights(cfg, seed=7)
    m = build(cfg, sd, dtype)
    rng = np.random.default_rng(11)
    reqs = {f"r{i}": prompt(cfg, n, seed=20 + i, sd=sd) for i, n in enumerate((130, 1, 64, 2, 65, 190, 33, 100, 7))}
    want = {r: Expected(sd, cfg, t) for r, t in reqs.items()}
    run = vn.StepRunner(m, max_batch=3, max_seq=192, pool_tokens=448)
    at = {r: 0 for r in reqs}
    waiting, live = list(reqs), []
    pages = {r: -(-len(t) // 64) for r, t in reqs.items()}
    while waiting or live:
        while waiting and len(live) < 3 and sum(pages[r] for r in live) + pages[waiting[0]] <= 7:
            live.append(waiting.pop(0))
        entries = []
        for r in live:
            left = len(reqs[r]) - at[r]
            n = min(left, int(rng.choice([0, 1, 1, 2, 3, 17, 64, 90])))
            if n:
                entries.append((r, reqs[r][at[r]:at[r] + n], list(range(n))))
        if not entries:
            continue
        got = run.step(entries).numpy()
        r0 = 0
        for r, t, _ in entries:
            want[r].check(got[r0:r0 + len(t)], dtype, slice(at[r], at[r] + len(t)), (r, at[r]))
            r0 += len(t)
            at[r] += len(t)
            if at[r] == len(reqs[r]):
                run.end(r)
                live.remove(r)
    m.check()
    assert run.cache.pages == (7, 7) and run.free_slots == 3


def test_a_batch_changes_nothing():
    """The same request alone and inside a batch: equal up to the order of sums (fp32 1e-5), every position."""
    cfg = BC.MODELS["plain"]
    sd = BC.weights(cfg)
    m = build(cfg, sd, "f32")
    a, b, c = prompt(cfg, 40, 1, sd), prompt(cfg, 90, 2, sd), prompt(cfg, 3, 3, sd)
    cache = m.new_cache(3, 128)
    got = m.forward_ragged(cache, [2, 0, 1], [40, 90, 3], np.concatenate([a, b, c]), range(133)).numpy()
    assert err(got[:40], whole(m, a)) < 1e-5 and err(got[40:130], whole(m, b)) < 1e-5 and err(got[130:], whole(m, c)) < 1e-5
    got = m.forward_ragged(cache, [0, 2], [1, 5], np.concatenate([a[:1], b[:5]]), [0, 5]).numpy()
    assert err(got[:1], whole(m, np.concatenate([b, a[:1]]))[-1:]) < 1e-5
    assert err(got[1:], whole(m, np.concatenate([a, b[:5]]))[-1:]) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(dtype):
    """Batches wide enough for the kernels' many-sequence shapes, as a prompt, as short portions that could be cut back, and
    as single tokens; more single tokens than the split-K route takes."""
    cfg = BC.config([M(heads=8, vdim=64, state=64, groups=2, mlp=E(ff=32)), A(heads=8, kv_heads=4, dim=64, vdim=64, rot=64, chunk=7, scale=0.15),
                     M(heads=10, vdim=128, state=72, groups=5, norm_groups=5), L(heads=8, dim=32, vdim=32, kv_rank=64, rot_dim=16, mlp=E(experts=5, identity=5, top=4))], width=64)
    sd = BC.weights(cfg, seed=15)
    m = build(cfg, sd, dtype)
    B, T = 40, 29
    checked = range(0, B, 13)
    toks = np.stack([prompt(cfg, T, seed=200 + b, sd=sd if b in checked else None) for b in range(B)])
    want = [Expected(sd, cfg, t) for t in toks[::13]]
    cache = m.new_cache(B, 32, max_pending=3)
    at, got = 0, []
    for n in (19, 2, 1, 3, 1, 3):
        got.append(m.forward_cached(toks[:, at:at + n], cache).numpy())
        cache.commit(n, np.full(B, n, np.int32))
        at += n
    got = np.concatenate(got, axis=1)
    for i, w in enumerate(want):
        w.check(got[13 * i], dtype)
    cache = m.new_cache(B, 32)
    got = m.forward_ragged(cache, list(range(B)), [T] * B, toks.reshape(-1), range(B * T)).numpy().reshape(B, T, -1)
    for i, w in enumerate(want):
        w.check(got[13 * i], dtype)
    B = 260
    cache = m.new_cache(B, 4)
    for t in range(3):
        rows = np.array([toks[b % 40, t] for b in range(B)])
        got = m.forward_ragged(cache, list(range(B)), [1] * B, rows, range(B)).numpy()
        for b in (0, 13, 253, 259):
            if b % 40 in checked:
                want[(b % 40) // 13].check(got[b:b + 1], dtype, slice(t, t + 1), (b, t))
    m.check()


def test_greedy_generation_through_the_scheduler():
    import versenext_b200 as vn
    cfg = BC.MODELS["plain"]
    sd = BC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    prompts = [prompt(cfg, n, seed=40 + n) for n in (20, 1, 70, 5)]
    want = [greedy(sd, cfg, p, 12) for p in prompts]
    assert [list(x) for x in m.generate(prompts, 12)] == want
    eng = vn.BatchEngine(m, max_batch=2, max_seq=128, pool_tokens=192, step_tokens=11)
    assert [list(x) for x in eng.run(prompts, 12)] == want
    assert eng.cache.pages == (3, 3)
    sampled = eng.run(prompts, 6, temperature=0.9, top_k=5, seed=3)
    assert [len(x) for x in sampled] == [6] * 4 and all(0 <= t < cfg["vocab"] for x in sampled for t in x)


def test_long_decoding():
    """Hundreds of single tokens: chunks have been left behind, states have been handed on at every step."""
    cfg = BC.MODELS["other_order"]
    sd = BC.weights(cfg, seed=12)
    toks = prompt(cfg, 420, sd=sd)
    want = Expected(sd, cfg, toks)
    for dtype in DTYPES:
        want.check(in_portions(build(cfg, sd, dtype), toks, [2] + [1] * 418), dtype)


@pytest.mark.parametrize("graph", [False, True])
def test_speculative_rounds_roll_states_back(graph):
    """A Bozasun model as target and another one as draft: the committed stream is the target's greedy stream, although most
    proposals are rejected and their states and convolution inputs dropped."""
    import versenext_b200 as vn
    cfg = BC.MODELS["plain"]
    sd = BC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    near = {n: bf16(a + 0.02 * np.random.default_rng(1).standard_normal(a.shape).astype(np.float32)) for n, a in sd.items()}
    prompts = np.stack([prompt(cfg, 9, seed=s) for s in (60, 61, 62)])
    want = [greedy(sd, cfg, p, 16) for p in prompts]
    for other in (near, BC.weights(cfg, seed=99)):
        d = build(cfg, other, "f32")
        for k in (1, 4):
            eng = vn.SpecEngine(m, d, max_batch=3, max_seq=64, k=k, graph=graph)
            out, stats = eng.generate(prompts, 16)
            assert [list(r) for r in out[:, 9:]] == want, k


def test_mechanisms_in_other_arrangements():
    """The parts are not tied to one design: norms of the heads with half-split pairs, chunks inside a window, an output gate
    and no biases; a latent with a rotated part, a window, sinks and a gate per head; a mixture of GELU experts without
    corrections; weights around zero."""
    import versenext_b200 as vn
    D, V, eps, T, F = 48, 60, 1e-4, 50, np.float64
    rng = np.random.default_rng(3)
    w = lambda *s: bf16((rng.standard_normal(s) / np.sqrt(s[-1])).astype(np.float32))
    rope = {"dims": 8, "base": 300.0}
    cfg = {"vocab_size": V, "dim": D, "norm_eps": eps, "token_side": 6, "layers": [
        {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.3, "window": 11, "chunk": 16, "qk_norm": True, "output_gate": True,
         "rope": rope, "mlp_hidden": 20, "mlp_act": "gelu_tanh", "experts": {"count": 5, "identity": 1, "top": 2}},
        {"mixer": "latent_attention", "heads": 3, "dim": 10, "rot_dim": 8, "vdim": 6, "kv_rank": 14, "scale": 0.4, "window": 9, "rope": dict(rope, interleaved=True),
         "mlp_hidden": 40, "mlp_act": "silu"}]}
    sd = {"embed": w(V, D) * 4, "head": w(V, D), "final.norm": w(D), "side.embed": w(V, 12) * 3}
    for i in range(2):
        sd.update({f"l{i}.norm1": w(D), f"l{i}.norm2": w(D), f"l{i}.side.gate": w(6, D), f"l{i}.side.proj": w(D, 6), f"l{i}.side.norm": 1 + w(D)})
    sd.update({"l0.mix.q": w(48, D) * 2, "l0.mix.k": w(24, D) * 2, "l0.mix.v": w(24, D), "l0.mix.g": w(48, D), "l0.mix.o": w(D, 48), "l0.mix.q.norm": 1 + w(12),
               "l0.mix.k.norm": 1 + w(12), "l0.mlp.router": w(6, D) * 2})
    for e in range(5):
        sd.update({f"l0.mlp.e{e}.gate": w(20, D) * 2, f"l0.mlp.e{e}.up": w(20, D) * 2, f"l0.mlp.e{e}.down": w(D, 20) * 2})
    sd.update({"l1.mix.q": w(54, D) * 2, "l1.mix.dkv": w(22, D), "l1.mix.dkv.norm": 1 + w(14), "l1.mix.uk": w(30, 14), "l1.mix.uv": w(18, 14), "l1.mix.sink": w(3) * 2,
               "l1.mix.g": w(3, D) * 2, "l1.mix.o": w(D, 18), "l1.mlp.gate": w(40, D), "l1.mlp.up": w(40, D), "l1.mlp.down": w(D, 40)})
    sd = {n: bf16(np.asarray(a, np.float32)) for n, a in sd.items()}
    W = {n: a.astype(F) for n, a in sd.items()}
    toks = rng.integers(0, V, T)
    from oracle import musutar as OM

    def half_split(x):
        return OM.rotate(x, rope)
    x = W["embed"][toks]
    h = OF.norm(x, W["l0.norm1"], eps)
    q = half_split(OB.norm((h @ W["l0.mix.q"].T).reshape(T, 4, 12), W["l0.mix.q.norm"], eps))
    k = half_split(OB.norm((h @ W["l0.mix.k"].T).reshape(T, 2, 12), W["l0.mix.k.norm"], eps))
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    o = OB.softmax_attention(q, k, (h @ W["l0.mix.v"].T).reshape(T, 2, 12), 0.3, OB.same_chunk(T, 16) & (i - j < 11))
    x = x + (o.reshape(T, 48) * OB.sigmoid(h @ W["l0.mix.g"].T)) @ W["l0.mix.o"].T
    h = OF.norm(x, W["l0.norm2"], eps)
    chosen, weight = OB.route(h @ W["l0.mlp.router"].T, np.zeros(6), 2, 1, 1)
    y = np.zeros_like(x)
    for t in range(T):
        for e, f in zip(chosen[t], weight[t]):
            g = {p: W[f"l0.mlp.e{e}.{p}"] for p in ("gate", "up", "down")} if e < 5 else None
            y[t] += f * (h[t] if g is None else (OB.gelu_tanh(h[t] @ g["gate"].T) * (h[t] @ g["up"].T)) @ g["down"].T)
    x = x + y
    side = lambda x, n: OB.side_input(x, W["side.embed"][toks, 6 * n:6 * n + 6], {k[3:]: a for k, a in W.items() if k.startswith(f"l{n}.")}, eps)
    x = x + side(x, 0)
    h = OF.norm(x, W["l1.norm1"], eps)
    q = (h @ W["l1.mix.q"].T).reshape(T, 3, 18)
    down = h @ W["l1.mix.dkv"].T
    c = OB.norm(down[:, :14], W["l1.mix.dkv.norm"], eps)
    k = np.concatenate([(c @ W["l1.mix.uk"].T).reshape(T, 3, 10), np.repeat(OB.rotate(down[:, None, 14:], rope), 3, 1)], 2)
    q = np.concatenate([q[..., :10], OB.rotate(q[..., 10:], rope)], 2)
    v = (c @ W["l1.mix.uv"].T).reshape(T, 3, 6)
    gate = OB.sigmoid(h @ W["l1.mix.g"].T)
    o = np.zeros((T, 3, 6))
    for a in range(3):
        s = np.where((j <= i) & (i - j < 9), q[:, a] @ k[:, a].T * 0.4, -np.inf)
        e = np.exp(s)
        o[:, a] = (e @ v[:, a]) / (e.sum(1) + np.exp(W["l1.mix.sink"][a]))[:, None] * gate[:, a:a + 1]
    x = x + o.reshape(T, 18) @ W["l1.mix.o"].T
    h = OF.norm(x, W["l1.norm2"], eps)
    x = x + (OB.silu(h @ W["l1.mlp.gate"].T) * (h @ W["l1.mlp.up"].T)) @ W["l1.mlp.down"].T
    x = x + side(x, 1)
    want = OF.norm(x, W["final.norm"], eps) @ W["head"].T
    m = vn.ComposedLM(cfg, dtype="f32")
    m.load_state_dict(sd)
    assert err(whole(m, toks), want) < 3e-5 and err(in_portions(m, toks, [20, 1, 2]), want) < 3e-5


def test_loading_is_checked():
    import versenext_b200 as vn
    cfg = BC.MODELS["plain"]
    sd = BC.weights(cfg)
    m = vn.BozasunLM(cfg, {n: a.shape for n, a in sd.items()}, dtype="f32")
    for n in list(sd)[:-1]:
        m.load_tensor(n, sd[n])
    with pytest.raises(ValueError):
        m.finalize()
    for name, a in (("l1.mlp.e7.gate", sd["l1.mlp.e0.gate"]), ("l3.mlp.up", sd["l0.mlp.up"]), ("l2.mix.sink", np.zeros(3, np.float32)),
                    ("l1.mix.in", sd["l1.mix.in"][:-1]), ("side.embed", sd["side.embed"][:, :-1]), ("l2.mix.dkv", sd["l2.mix.dkv"][:-2])):
        with pytest.raises(ValueError):
            m.load_tensor(name, a)
    m.load_tensor(list(sd)[-1], sd[list(sd)[-1]])
    m.finalize()
    toks = prompt(cfg, 10)
    assert err(whole(m, toks), OB.forward(sd, cfg, toks)) < 3e-5
    for layer, part, bad in ((0, "mixer", {"heads": 3}), (0, "mixer", {"rot": {"base": 10.0, "dims": 26}}), (1, "mixer", {"groups": 4}), (1, "mixer", {"norm_groups": 7}),
                             (2, "mixer", {"rot_dim": 10}), (2, "mixer", {"rot": None}), (1, "mlp", {"router": dict(cfg["layers"][1]["mlp"]["router"], top=5)}),
                             (1, "mlp", {"router": dict(cfg["layers"][1]["mlp"]["router"], identity=4)})):
        other = json.loads(json.dumps(cfg))
        other["layers"][layer][part].update(bad)
        with pytest.raises(ValueError):
            vn.BozasunLM(other, {}, dtype="f32")


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_and_command_line(tmp_path, dtype):
    cfg = BC.MODELS["other_order"]
    sd = BC.weights(cfg, seed=13)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir()
    out.mkdir()
    write_model(model, cfg, sd)
    a, b, c = prompt(cfg, 80, 1, sd).tolist(), prompt(cfg, 30, 2, sd).tolist(), prompt(cfg, 5, 3, sd).tolist()
    steps = [([("a", a[:70], [0, 69])], []), ([("a", a[70:71], [0]), ("b", b[:20], [19])], []), ([("b", b[20:], [])], ["b"]),
             ([("c", c, [4]), ("a", a[71:], [8])], ["a", "c"]), ([("b2", b, [29])], ["b2"])]
    text = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in e], "end": end}) + "\n"
                   for i, (e, end) in enumerate(steps))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "192"], input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not (out / "2.f32").exists()
    EA, EB, EC = (Expected(sd, cfg, t) for t in (a, b, c))
    want = {0: [(EA, 0), (EA, 69)], 1: [(EA, 70), (EB, 19)], 3: [(EC, 4), (EA, 79)], 4: [(EB, 29)]}
    for i, rows in want.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert len(got) == len(rows)
        for g, (e, p) in zip(got, rows):
            e.check(g[None], "bf16" if dtype == "bfloat16" else "f32", slice(p, p + 1), (i, p))
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "versenext_b200", "generate", "--model", str(model), "--dtype", "f32", "--prompt",
                            ",".join(map(str, c)), "--max-new-tokens", "5"], capture_output=True, text=True, timeout=300, cwd=root)
        assert r.returncode == 0, r.stderr
        assert json.loads(r.stdout.splitlines()[-1]) == greedy(sd, cfg, c, 5)
