"""Test bodies for the Busavik decoder that run the same way on the CPU stand-in of the kernel layer and on the
GPU: each takes ``make_engine(cfg_dict, tensors, **kw)`` and a band (how close the engine has to be), and compares
the engine with the plain implementation in float64."""
from __future__ import annotations

import copy

import torch

import plain_busavik as plain
from safuvik_tiny import tokens_for, run_cut, rel_err
from vaderax_cases import Band                                     # the same measure of closeness
from busavik_tiny import CONFIGS, make_tensors, model, latent_layer
from rbitnet_b200.engine.step import StepEntry


def reference(cfg, tensors, tokens):
    return plain.forward(cfg, tensors, tokens, torch.float64)


def whole(make_engine, name, band, n=150):
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=11, spread=band.spread)
    toks = tokens_for(cfg, n, 5)
    assert band.ok(run_cut(make_engine(cfg, tensors), toks, []), reference(cfg, tensors, toks))


def prefill_against_decoding(make_engine, name, band, n=90, prompt=37):
    """A prompt in one step and the rest token by token, and everything token by token, against the whole."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=12, spread=band.spread)
    toks = tokens_for(cfg, n, 6)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    assert band.ok(run_cut(eng, toks, list(range(prompt, n))), ref)
    assert band.ok(run_cut(eng, toks, list(range(1, n))), ref)


def portions(make_engine, name, band, n=140):
    """Portions of 2 tokens, of a page, of odd sizes, and a last portion of one token."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=13, spread=band.spread)
    toks = tokens_for(cfg, n, 7)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    for cuts in (list(range(2, n, 2)), [64, 128], [3, 8, 9, 63, 65, 127, n - 1], [1, 2, 4, 70], [1, 3, 4, 5, 66, 67, 69]):
        assert band.ok(run_cut(eng, toks, cuts), ref), cuts


def batches_against_alone(make_engine, name, band, lengths=(1, 2, 75, 9, 131), decode=12):
    """Unequal prompts in one step, then decoded together, the shorter requests ending earlier; the slots and pages of
    those that ended are used again by a second batch.  Against each request alone (plain model)."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=14, spread=band.spread)
    eng = make_engine(cfg, tensors, max_tokens=64 * 8)
    for round_ in range(2):
        reqs = [tokens_for(cfg, n + (decode if i % 2 else decode // 2), 20 + 10 * round_ + i) for i, n in enumerate(lengths)]
        refs = [reference(cfg, tensors, r) for r in reqs]
        slots = [eng.new_sequence() for _ in reqs]
        got = [[] for _ in reqs]
        out = eng.step([StepEntry(s, r[:n], list(range(n))) for s, r, n in zip(slots, reqs, lengths)])
        at = 0
        for i, n in enumerate(lengths):
            got[i].append(out[at:at + n])
            at += n
        fed = list(lengths)
        live = list(range(len(reqs)))
        while live:
            out = eng.step([StepEntry(slots[i], [reqs[i][fed[i]]], [0]) for i in live])
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
                fed[i] += 1
            for i in [i for i in live if fed[i] == len(reqs[i])]:
                eng.end_sequence(slots[i])
                live.remove(i)
        assert band.ok_all([(torch.cat(got[i]).float().cpu(), refs[i]) for i in range(len(reqs))]), round_


def slots_and_pages_used_again(make_engine, name, band):
    """A cache of three pages: every sequence gets the pages that the one before gave back; nothing of the
    earlier sequence may show."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=15, spread=band.spread)
    eng = make_engine(cfg, tensors, max_tokens=64 * 3)
    for k, n in enumerate((130, 70, 150, 5, 129)):
        toks = tokens_for(cfg, n, 40 + k)
        got = run_cut(eng, toks, [n // 2, n - 3, n - 2, n - 1])
        assert band.ok(got, reference(cfg, tensors, toks)), k


def long_decoding(make_engine, name, band, n=200, prompt=3):
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=16, spread=band.spread)
    toks = tokens_for(cfg, n, 8)
    assert band.ok(run_cut(make_engine(cfg, tensors), toks, list(range(prompt, n))), reference(cfg, tensors, toks))


def first_tokens(make_engine, name, band):
    """Sequences of one to five tokens, whole and token by token."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=17, spread=band.spread)
    eng = make_engine(cfg, tensors)
    pairs = []
    for n in (1, 2, 3, 4, 5):
        toks = tokens_for(cfg, n, 50 + n)
        ref = reference(cfg, tensors, toks)
        pairs += [(run_cut(eng, toks, []), ref), (run_cut(eng, toks, list(range(1, n))), ref)]
    assert band.ok_all(pairs)


def random_configuration(make_engine, seed, band, n=100):
    """A configuration drawn from ``seed``: whole, the last tokens one by one, and two unequal requests together."""
    from busavik_tiny import random_config
    cfg = random_config(seed)
    tensors = make_tensors(cfg, seed=seed, spread=band.spread)
    toks = tokens_for(cfg, n, seed)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    assert band.ok(run_cut(eng, toks, []), ref), cfg
    assert band.ok(run_cut(eng, toks, [70] + list(range(90, n))), ref), cfg
    other = tokens_for(cfg, 31, seed + 1)
    slots = [eng.new_sequence(), eng.new_sequence()]
    out = eng.step([StepEntry(slots[0], toks[:66], list(range(66))), StepEntry(slots[1], other[:29], list(range(29)))])
    got = [[out[:66]], [out[66:]]]
    for k in range(2):
        out = eng.step([StepEntry(slots[0], [toks[66 + k]], [0]), StepEntry(slots[1], [other[29 + k]], [0])])
        got[0].append(out[:1])
        got[1].append(out[1:])
    for s_ in slots:
        eng.end_sequence(s_)
    assert band.ok_all([(torch.cat(got[0]).float().cpu(), ref[:68]), (torch.cat(got[1]).float().cpu(), reference(cfg, tensors, other))]), cfg


def turned_part_decides(make_engine, tol, cuts, n=150, last=None):
    """One attention layer whose unturned scores are small beside the turned ones: what a position sees depends on the
    distances.  A wrong position, frequency or magnitude shows; sequences run past the scaling's `original`.  ``last``:
    only that many last positions are compared."""
    scaling = (4.0, 24, 8.0, 1.0)
    cfg = model(40, 32, [latent_layer(2, 8, 16, 8, 24, 16, 0.4, None, base=200.0, scaling=scaling)])
    tensors = make_tensors(cfg, seed=27)
    H, D, R = 2, 8, 16
    uq = tensors["l0.mix.uq"].view(H, D + R, -1).clone()
    uq[:, :D] *= 0.125
    uq[:, D:] *= 2.0
    tensors["l0.mix.uq"] = uq.reshape(H * (D + R), -1)
    tensors["l0.mix.dkv"][16:] *= 2.0
    toks = tokens_for(cfg, n, 12)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    pick = (lambda x: x[-last:]) if last else (lambda x: x)
    assert rel_err(pick(run_cut(eng, toks, cuts)), pick(ref)) <= tol
    # what the frequencies and their scaling do is far outside the tolerance
    for other in (None, (4.0, 24, 8.0, 2.0), (2.0, 24, 8.0, 1.0)):
        bent = copy.deepcopy(cfg)
        bent["layers"][0] = latent_layer(2, 8, 16, 8, 24, 16, 0.4, None, base=200.0, scaling=other)
        assert rel_err(pick(reference(bent, tensors, toks)), pick(ref)) > 3.0 * tol, other


def one_far_key_stands_out(make_engine, tol, n, far, cuts, last_only=False, kv_rank=16):
    """One attention layer.  Position ``far`` holds a token that occurs nowhere else, and the last token's query is made
    to point at that token's key, far above every other score; the turned parts are small.  The last logits then carry the
    far position's latent: the engine must agree with the plain model, and exchanging the far token must move them a
    lot.  ``last_only``: only the last position is compared (in bfloat16 the sharp scores of the others, which nothing
    here arranges, amplify rounding)."""
    H, D, R, C = 2, 16, 8, kv_rank
    cfg = model(40, 32, [latent_layer(H, D, R, 8, C, C, 1.0, None)], logit_scale=1.0)
    tensors = make_tensors(cfg, seed=23)
    V = cfg["vocab"]
    toks = [1 + (i * 7) % (V - 3) for i in range(n)]
    toks[far] = V - 1
    toks[-1] = V - 2
    # The last token's embedding is the far token's with its values permuted; the queries' way through their latent is
    # the keys' way with the first matrix's columns permuted alike, and the curve before the two is the same on every
    # channel.  So the unturned q(last) is k(far), and their score |k|^2.
    perm = torch.randperm(cfg["width"], generator=torch.Generator().manual_seed(5))
    emb, dkv = tensors["embed"], tensors["l0.mix.dkv"]
    emb[V - 2] = emb[V - 1][perm]
    tensors["l0.norm1"], tensors["l0.norm1.b"] = torch.ones(cfg["width"]), torch.zeros(cfg["width"])
    dkv[C:] *= 0.05
    tensors["l0.mix.dq"] = dkv[:C][:, perm].clone()
    tensors["l0.mix.dq.norm"] = tensors["l0.mix.dkv.norm"].clone()
    uq = tensors["l0.mix.uq"].view(H, D + R, C).clone()
    uq[:, :D] = tensors["l0.mix.uk"].view(H, D, C)
    uq[:, D:] *= 0.05
    tensors["l0.mix.uq"] = uq.reshape(H * (D + R), C)
    tensors = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in tensors.items()}
    # sharp: the far key's score is 60, the others' a fraction of it
    t = {k: v.double() for k, v in tensors.items()}
    c = plain.rms(torch.tanh(t["l0.norm1.alpha"] * t["embed"][V - 1]) @ t["l0.mix.dkv"][:C].T, cfg["norm"]["eps"]) * t["l0.mix.dkv.norm"]
    cfg["layers"][0]["mixer"]["scale"] = 60.0 / float(((t["l0.mix.uk"] @ c).view(H, D) ** 2).sum(-1).min())
    ref = reference(cfg, tensors, toks)
    other = list(toks)
    other[far] = 2
    ref_other = reference(cfg, tensors, other)
    assert float((ref[-1] - ref_other[-1]).abs().max() / ref[-1].abs().max()) > 3.0 * tol, "the far key does not stand out"
    eng = make_engine(cfg, tensors)
    pick = (lambda x: x[-1:]) if last_only else (lambda x: x)
    assert rel_err(pick(run_cut(eng, toks, cuts)), pick(ref)) <= tol
    assert rel_err(pick(run_cut(eng, other, cuts)), pick(ref_other)) <= tol


def greedy_generation(make_engine, name, prompts=(7, 1, 30), new=24):
    """``Engine.generate`` (scheduler, batches, the captured decode step where there is one) against a greedy loop
    over the plain model."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=21)
    eng = make_engine(cfg, tensors, graphs=True)
    ps = [tokens_for(cfg, n, 60 + i) for i, n in enumerate(prompts)]
    results = eng.generate(ps, max_tokens=new, temperature=0.0, stop_ids=[])
    for p, r in zip(ps, results):
        seq = list(p)
        for step, tok in enumerate(r.tokens):
            logits = reference(cfg, tensors, seq)[-1]
            best = int(torch.argmax(logits))
            if best != tok:
                # a tie within rounding is not a fault; anything else is
                assert float(logits[best] - logits[tok]) <= 1e-4 * float(logits.abs().max()), (step, best, tok)
            seq.append(tok)
        assert len(r.tokens) == new
