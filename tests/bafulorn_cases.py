"""Test bodies for the Bafulorn decoder that run the same way on the CPU stand-in of the kernel layer and on the
GPU: each takes ``make_engine(cfg_dict, tensors, **kw)`` and a band (how close the engine has to be), and compares
the engine with the plain implementation in float64."""
from __future__ import annotations

import torch

import plain_bafulorn as plain
from safuvik_tiny import tokens_for, run_cut, rel_err
from vaderax_cases import Band                                     # the same measure of closeness
from bafulorn_tiny import CONFIGS, make_tensors, model, latent_layer, attention_layer, mamba_layer
from rbitnet_b200.engine.step import StepEntry


def reference(cfg, tensors, tokens):
    return plain.forward(cfg, tensors, tokens, torch.float64)


def whole(make_engine, name, band, n=200):
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=11, spread=band.spread)
    toks = tokens_for(cfg, n, 5)
    assert band.ok(run_cut(make_engine(cfg, tensors), toks, []), reference(cfg, tensors, toks))


def prefill_against_decoding(make_engine, name, band, n=100, prompt=37):
    """A prompt in one step and the rest token by token, and everything token by token, against the whole."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=12, spread=band.spread)
    toks = tokens_for(cfg, n, 6)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    assert band.ok(run_cut(eng, toks, list(range(prompt, n))), ref)
    assert band.ok(run_cut(eng, toks, list(range(1, n))), ref)


def portions(make_engine, name, band, n=150):
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
    """A cache of three pages: every sequence gets the slot, the pages and the state that the one before gave back; nothing
    of the earlier sequence may show."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, seed=15, spread=band.spread)
    eng = make_engine(cfg, tensors, max_tokens=64 * 3)
    for k, n in enumerate((130, 70, 150, 5, 129)):
        toks = tokens_for(cfg, n, 40 + k)
        got = run_cut(eng, toks, [n // 2, n - 3, n - 2, n - 1])
        assert band.ok(got, reference(cfg, tensors, toks)), k


def long_decoding(make_engine, name, band, n=210, prompt=3):
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
    from bafulorn_tiny import random_config
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


def _last_and_far(kind, n, far, window, keep, kv_rank, dim, sharp=60.0):
    """(cfg, tensors, tokens): one attention layer.  Position ``far`` holds a token that occurs nowhere else, and the last
    token's query is made to point at that token's key, far above every other score."""
    E, H = 32, 2
    layer = latent_layer(H, dim, 8, kv_rank, window, 1.0) if kind == "latent" else attention_layer(H, H, dim, window, keep, 1.0, dim // 4)
    cfg = model(40, E, [layer], mult=1.0)
    t = make_tensors(cfg, seed=23)
    V = cfg["vocab"]
    toks = [1 + (i * 7) % (V - 3) for i in range(n)]
    toks[far], toks[-1] = V - 1, V - 2
    # The last token's embedding is the far token's with its values permuted, the queries read permuted columns, and the
    # norms before them weigh every channel alike: so the last query is the far key (but for the latent's norm, a factor).
    perm = torch.randperm(E, generator=torch.Generator().manual_seed(5))
    t["embed"][V - 2] = t["embed"][V - 1][perm]
    t["embed.norm"], t["l0.norm1"] = torch.zeros(E), torch.zeros(E)
    if kind == "latent":
        t["l0.mix.q"] = (t["l0.mix.uk"] * t["l0.mix.dkv.norm"]) @ t["l0.mix.dkv"][:, perm]
    else:
        k = t["l0.mix.k"].view(H, dim, E).clone()
        k[:, :dim // 4] *= 0.05                                  # the turned values weigh little: distances do not matter
        t["l0.mix.k"] = k.reshape(H * dim, E)
        t["l0.mix.k.b"] = t["l0.mix.k.b"] * 0.1
        t["l0.mix.q"], t["l0.mix.q.b"] = t["l0.mix.k"][:, perm].clone(), t["l0.mix.k.b"].clone()
    t = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in t.items()}
    d = {k: v.double() for k, v in t.items()}
    eps = cfg["norm"]["eps"]
    h = plain.norm(plain.norm(d["embed"], d["embed.norm"], eps), d["l0.norm1"], eps)
    if kind == "latent":
        key = (plain.rms(h[V - 1] @ d["l0.mix.dkv"].T, eps) * d["l0.mix.dkv.norm"]) @ d["l0.mix.uk"].T
        query = h[V - 2] @ d["l0.mix.q"].T
    else:
        key = h[V - 1] @ d["l0.mix.k"].T + d["l0.mix.k.b"]
        query = h[V - 2] @ d["l0.mix.q"].T + d["l0.mix.q.b"]
    cfg["layers"][0]["mixer"]["scale"] = sharp / float((key * query).view(H, dim).sum(-1).min())
    return cfg, t, toks


def one_key_stands_out(make_engine, tol, kind, n, far, window, keep, seen, cuts, last_only=False, kv_rank=16, dim=16):
    """The last logits carry the far position's value where the mask lets the last position see it (``seen``) and nothing
    of it where not: the engine agrees with the plain model, and exchanging the far token moves the last logits a lot, or
    not at all.  ``last_only``: only the last position is compared (in bfloat16 the sharp scores of the others, which
    nothing here arranges, amplify rounding)."""
    cfg, tensors, toks = _last_and_far(kind, n, far, window, keep, kv_rank, dim)
    other = list(toks)
    other[far] = 2
    ref, ref_other = reference(cfg, tensors, toks), reference(cfg, tensors, other)
    moved = float((ref[-1] - ref_other[-1]).abs().max() / ref[-1].abs().max())
    assert (moved > 3.0 * tol) if seen else (moved == 0.0), moved
    eng = make_engine(cfg, tensors)
    pick = (lambda x: x[-1:]) if last_only else (lambda x: x)
    assert rel_err(pick(run_cut(eng, toks, cuts)), pick(ref)) <= tol
    assert rel_err(pick(run_cut(eng, other, cuts)), pick(ref_other)) <= tol


#: (length, far position, window, kept positions, whether the last position sees it): keys far away, at page borders, just
#: inside and just outside a window, the last kept position and the one after it
KEYS = [(300, 299 - 90, 91, 0, True), (300, 299 - 91, 91, 0, False), (200, 199 - 63, 64, 0, True), (200, 199 - 64, 64, 0, False),
        (260, 128, 132, 0, True), (260, 127, 132, 0, False), (300, 2, None, 0, True), (700, 63, None, 0, True)]
KEPT_KEYS = [(300, 9, 50, 10, True), (300, 10, 50, 10, False), (300, 0, 50, 1, True), (300, 1, 50, 1, False), (200, 63, 20, 64, True),
             (200, 64, 20, 64, False), (330, 69, 64, 70, True), (330, 70, 64, 70, False), (190, 130, 60, 7, True), (190, 129, 60, 7, False),
             (700, 5, 100, 6, True), (260, 128, 64, 129, True), (100, 3, 1, 4, True), (100, 98, 1, 4, False)]


def state_carries_the_first_token(make_engine, tol, cuts, n=400):
    """One state-space layer that hardly forgets and whose state only the first token writes much into: the last logits
    still carry it."""
    cfg = model(40, 32, [mamba_layer(2, 16, 24, 1, 4, 1, None)], mult=1.0)
    t = make_tensors(cfg, seed=29)
    t["l0.mix.A_log"] = torch.full((2,), -9.0)
    rows = t["l0.mix.in"].shape[0]
    t["embed.norm"], t["l0.norm1"] = torch.zeros(32), torch.zeros(32)
    toks = [1 + (i * 7) % 37 for i in range(n)]
    toks[0] = 39
    # dt is large where channel 0 of the row is, which only the first token's is
    t["embed"][:, 0] = -0.05
    t["embed"][39] *= 0.1
    t["embed"][39, 0] = 0.2
    t["l0.mix.in"][rows - 2:] = 0.0
    t["l0.mix.in"][rows - 2:, 0] = 2.0
    t["l0.mix.dt_bias"] = torch.full((2,), -6.0)
    t["l0.mix.D"] *= 0.05
    t = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in t.items()}
    other = list(toks)
    other[0] = 5
    ref, ref_other = reference(cfg, t, toks), reference(cfg, t, other)
    assert float((ref[-1] - ref_other[-1]).abs().max() / ref[-1].abs().max()) > 10.0 * tol
    eng = make_engine(cfg, t)
    assert rel_err(run_cut(eng, toks, cuts), ref) <= tol
    assert rel_err(run_cut(eng, other, cuts), ref_other) <= tol


def turned_part_decides(make_engine, tol, cuts, n=150, last=None):
    """One attention layer whose unturned scores are small beside the turned ones: what a position sees depends on the
    distances.  A wrong position, frequency or pairing shows; sequences run past the scaling's `original`.  ``last``:
    only that many last positions are compared."""
    scaling = (4.0, 1.0, 4.0, 48)

    def layer(sc, base=60.0):
        return attention_layer(2, 1, 16, 100, 3, 0.4, 12, None, base=base, scaling=sc)
    cfg = model(40, 32, [layer(scaling)], mult=1.0)
    tensors = make_tensors(cfg, seed=27)
    toks = tokens_for(cfg, n, 12)
    ref = reference(cfg, tensors, toks)
    eng = make_engine(cfg, tensors)
    pick = (lambda x: x[-last:]) if last else (lambda x: x)
    assert rel_err(pick(run_cut(eng, toks, cuts)), pick(ref)) <= tol
    for other in (layer(None), layer((4.0, 1.0, 2.0, 48)), layer((2.0, 1.0, 4.0, 48)), layer((4.0, 1.0, 4.0, 100)), layer(scaling, 80.0)):
        assert rel_err(pick(reference(model(40, 32, [other], mult=1.0), tensors, toks)), pick(ref)) > 2.0 * tol, other


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
