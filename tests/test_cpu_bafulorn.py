"""The Bafulorn decoder through the package's host logic (configuration, parts, cache manager, step function, scheduler,
generation, trace replay) on the CPU stand-in of the kernel layer, against the plain implementation."""
import json
import math

import pytest
import torch

import plain_bafulorn as plain
import bafulorn_cases as cases
from safuvik_tiny import write_model, tokens_for
from bafulorn_tiny import CONFIGS, make_tensors, spec_of
from torch_ops import TorchOps
from rbitnet_b200.config import config_from_dict, ConfigError, load_config
from rbitnet_b200.engine import Engine

# float32 against float64 on weights that are scaled up so that faults show
TOL = 2e-4
BAND = cases.Band(TOL)


def make_engine(cfg, tensors, max_tokens=64 * 16, graphs=False, **kw):
    return Engine(config_from_dict(cfg), dict(tensors), dtype="float32", ops=TorchOps(torch.float32),
                  max_tokens=max_tokens, max_seq=1024, **kw)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole(name):
    cases.whole(make_engine, name, BAND, n=140)


@pytest.mark.parametrize("name", ["A", "B"])
def test_prefill_against_decoding(name):
    cases.prefill_against_decoding(make_engine, name, BAND, n=40, prompt=13)


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_random_configurations(seed):
    cases.random_configuration(make_engine, seed, BAND, n=100)


def test_portions():
    cases.portions(make_engine, "B", BAND, n=132)


def test_batches():
    cases.batches_against_alone(make_engine, "A", BAND, lengths=(1, 2, 67, 9), decode=6)


def test_slots_and_pages_used_again():
    cases.slots_and_pages_used_again(make_engine, "A", BAND)


def test_first_tokens():
    cases.first_tokens(make_engine, "D", BAND)


@pytest.mark.parametrize("n,far,window,keep,seen", cases.KEYS[:7])
def test_one_key_of_the_latent_attention(n, far, window, keep, seen):
    cases.one_key_stands_out(make_engine, TOL, "latent", n, far, window, keep, seen, cuts=[n - 40, n - 2, n - 1])


@pytest.mark.parametrize("n,far,window,keep,seen", cases.KEYS[:7] + [k for k in cases.KEPT_KEYS if k[0] < 700])
def test_one_key_of_the_attention(n, far, window, keep, seen):
    cases.one_key_stands_out(make_engine, TOL, "attention", n, far, window, keep, seen, cuts=[n - 40, n - 2, n - 1])


def test_state_carries_the_first_token():
    cases.state_carries_the_first_token(make_engine, TOL, cuts=[2, 100, 101, 180], n=200)


def test_turned_part():
    cases.turned_part_decides(make_engine, TOL, cuts=[40, 63, 64, 100], n=130)


def test_greedy_generation():
    cases.greedy_generation(make_engine, "A", prompts=(5, 1, 12), new=8)


# ---- every mechanism of the plain implementation against an independent statement of it
def test_plain_mask():
    see = plain.visible(9, {"size": 3, "keep_first": 2})
    for i in range(9):
        want = [j for j in range(9) if j in (i, i - 1, i - 2) or (j < 2 and j <= i)]
        assert see[i].nonzero().flatten().tolist() == want
    assert plain.visible(5, None).equal(torch.tril(torch.ones(5, 5, dtype=torch.bool)))
    assert plain.visible(6, {"size": 1}).equal(torch.eye(6, dtype=torch.bool))


def test_plain_rotation_and_stretched_frequencies():
    torch.manual_seed(1)
    x = torch.randn(5, 2, 7, dtype=torch.float64)
    y = plain.rotate(x, {"base": 100.0, "dims": 4})
    for t in range(5):
        for i, f in enumerate((1.0, 0.1)):
            c, s = math.cos(t * f), math.sin(t * f)
            assert torch.allclose(y[t, :, i], x[t, :, i] * c - x[t, :, i + 2] * s)
            assert torch.allclose(y[t, :, i + 2], x[t, :, i + 2] * c + x[t, :, i] * s)
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
    # base e^8 and 8 dims: pair i turns by e^(-2 i), its wavelength is 2 pi e^(2 i); original 2 pi e^3 puts the borders of
    # low = e^-2 and high = e at wavelengths 2 pi e^5 and 2 pi e^2: pair 0 stays, pair 3 is stretched, pairs 1 and 2 ...
    rot = {"base": math.exp(8.0), "dims": 8, "scaling": {"factor": 5.0, "original": 2 * math.pi * math.exp(3.0), "low": math.exp(-2.0),
                                                         "high": math.exp(0.5)}}
    low, high = math.exp(-2.0), math.exp(0.5)
    s = (math.exp(3.0) / math.exp(4.0) - low) / (high - low)         # pair 2 lies between, e^(3 - 4) turns in `original`
    want = [1.0, math.exp(-2.0), math.exp(-4.0) * ((1 - s) / 5.0 + s), math.exp(-6.0) / 5.0]
    assert torch.allclose(plain.frequencies(rot), torch.tensor(want).double())


def test_plain_attention_and_feed_forward_pieces():
    torch.manual_seed(0)
    q, k, v = torch.randn(6, 4, 3).double(), torch.randn(6, 2, 3).double(), torch.randn(6, 2, 5).double()
    out = plain.softmax_attention(q, k, v, 0.7, plain.visible(6, {"size": 2, "keep_first": 1}))
    for t in range(6):
        seen = sorted({0, max(t - 1, 0), t})
        for h in range(4):
            w = torch.exp(torch.stack([(q[t, h] @ k[j, h // 2]) * 0.7 for j in seen]))
            assert torch.allclose(out[t, h], (w[:, None] * v[seen, h // 2]).sum(0) / w.sum())
    z = torch.linspace(-4, 4, 9).double()
    assert torch.allclose(plain.silu(z), torch.nn.functional.silu(z)) and torch.allclose(plain.relu(z), torch.nn.functional.relu(z))
    assert torch.allclose(plain.softplus(10 * z), torch.nn.functional.softplus(10 * z))
    ids, weights = plain.choose(torch.tensor([0.5, 3.0, -1.0, 2.0]).double(), torch.tensor([0.0, -1.0, 0.9, 0.0]).double(), 2, 3.0)
    s = torch.sigmoid(torch.tensor([-1.0, 2.0]).double())
    assert ids.tolist() == [2, 3] and torch.allclose(weights, 3.0 * s / s.sum())
    x, w = torch.tensor([[3.0, -4.0]]).double(), torch.tensor([0.5, 0.0]).double()
    assert torch.allclose(plain.norm(x, w, 0.0), torch.tensor([[4.5, -4.0]]).double() / math.sqrt(12.5))


def test_plain_state_space_pieces():
    torch.manual_seed(2)
    T, H, P, G, N = 5, 4, 3, 2, 2
    x, B, C = torch.randn(T, H, P).double(), torch.randn(T, G, N).double(), torch.randn(T, G, N).double()
    dt, A, D = torch.rand(T, H).double() + 0.1, torch.randn(H).double(), torch.randn(H).double()
    y = plain.state_space(x, B, C, dt, A, D)
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                decay = math.exp(-math.exp(float(A[h])) * float(dt[j + 1:t + 1, h].sum()))
                want = want + decay * dt[j, h] * (C[t, h // 2] @ B[j, h // 2]) * x[j, h]
            assert torch.allclose(y[t, h], want)
    taps, bias = torch.randn(3, 2).double(), torch.randn(3).double()
    u = torch.randn(4, 3).double()
    conv = plain.causal_convolution(u, taps, bias)
    assert torch.allclose(conv[0], bias + taps[:, 1] * u[0]) and torch.allclose(conv[3], bias + taps[:, 1] * u[3] + taps[:, 0] * u[2])
    v = plain.gated_group_norm(u[:, :2], u[:, 1:], torch.tensor([2.0, 3.0]).double(), 2, 0.0)
    assert torch.allclose(v.abs(), torch.tensor([2.0, 3.0]).double().expand(4, 2))       # parts of one value: its sign remains


@pytest.mark.parametrize("what", ["head gate", "latent's norm", "kept positions", "window", "values before the rotation", "q's bias",
                                  "k's bias", "o's bias", "dt's bias", "own term", "convolution", "its bias", "norm in parts",
                                  "gate before the norm", "relu", "correction", "weights divided", "router scale", "shared expert",
                                  "result norm", "embedding norm", "residual_mult"])
def test_leaving_a_mechanism_out_shows(what, monkeypatch):
    """A mistake planted in the plain implementation moves its logits far outside the tolerance, so the tests that compare
    with it would see the same mistake in the package."""
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    tensors = make_tensors(cfg, 4)
    toks = tokens_for(cfg, 60, 2)
    ref = plain.forward(cfg, tensors, toks)
    bent = dict(tensors)

    def change(end, f):
        bent.update({k: f(v) for k, v in tensors.items() if k.endswith(end)})
    zero = {"head gate": "mix.g", "q's bias": "mix.q.b", "k's bias": "mix.k.b", "o's bias": "mix.o.b", "dt's bias": "dt_bias",
            "own term": "mix.D", "its bias": "conv.b", "result norm": "norm1b", "embedding norm": "embed.norm", "correction": "correction"}
    if what in zero:
        change(zero[what], lambda v: v * 0.0)
    elif what == "latent's norm":
        change("dkv.norm", torch.ones_like)
    elif what == "kept positions":
        cfg["layers"][0]["mixer"]["mask"]["keep_first"] -= 1
    elif what == "window":
        cfg["layers"][2]["mixer"]["mask"]["size"] += 1
    elif what == "values before the rotation":
        rotate = plain.rotate
        monkeypatch.setattr(plain, "softmax_attention", lambda q, k, v, scale, see, f=plain.softmax_attention:
                            f(q, k, k if v.shape == k.shape else v, scale, see))
        assert rotate is plain.rotate
    elif what == "convolution":
        change("mix.conv", lambda v: torch.cat([v[:, :1] * 0.0, v[:, 1:]], dim=1))
    elif what == "norm in parts":
        cfg["layers"][1]["mixer"]["norm_groups"] = 1
    elif what == "gate before the norm":
        monkeypatch.setattr(plain, "gated_group_norm", lambda y, z, w, groups, eps: plain.rms(
            y.view(y.shape[0], groups, -1), eps).reshape(y.shape) * w * plain.silu(z))
    elif what == "relu":
        monkeypatch.setattr(plain, "relu", plain.silu)
    elif what == "weights divided":
        def undivided(z, correction, top, scale):
            s = torch.sigmoid(z)
            ids = torch.argsort(s + correction, descending=True, stable=True)[:top]
            return ids, s[ids] * scale
        monkeypatch.setattr(plain, "choose", undivided)
    elif what == "router scale":
        cfg["layers"][1]["mlp"]["router"]["scale"] = 1.0
    elif what == "shared expert":
        cfg["layers"][1]["mlp"].pop("shared")
    else:
        cfg["residual_mult"] = 0.45
    assert cases.rel_err(plain.forward(cfg, bent, toks), ref) > 10 * TOL


def test_caches_states_and_what_a_window_keeps():
    """What every layer asks for; pages behind a window come back, those of the kept positions stay."""
    cfg = CONFIGS["C"]
    eng = make_engine(cfg, make_tensors(cfg, 1))
    caches, _, states = eng.model.cache_plan()
    assert set(caches) == {1, 2, 3, 4} and set(states) == {0}
    assert caches[1].streams == ((1, 128),) and (caches[1].window, caches[1].keep_first) == (65, 0)
    assert (caches[2].window, caches[2].keep_first) == (64, 70) and caches[3].window is None
    assert states[0]["S"].shape == (8, 64, 32) and states[0]["tail"].shape == (4, 8 * 32 + 2 * 2 * 64)
    slot = eng.new_sequence()
    eng.step([cases.StepEntry(slot, tokens_for(cfg, 400, 1), [])])
    held = {(g.need.window, g.need.keep_first): [i for i, p in enumerate(pages) if p >= 0]
            for g, pages in zip(eng.cache.groups, eng.cache.book.pages[slot])}
    assert held[(64, 70)] == [0, 1, 5, 6] and held[(65, 0)] == [5, 6] and held[(None, 0)] == list(range(7))
    free = [p.n_free for p in eng.cache.book.pools]
    eng.end_sequence(slot)
    assert [p.n_free - f for p, f in zip(eng.cache.book.pools, free)] == [
        len(held[(g.need.window, g.need.keep_first)]) for g in eng.cache.groups]


def test_residual_after_every_layer():
    import numpy as np
    from rbitnet_b200.engine.step import build_meta, SeqChunk, StepContext
    cfg = CONFIGS["A"]
    tensors = make_tensors(cfg, 2)
    toks = tokens_for(cfg, 19, 3)
    eng = make_engine(cfg, tensors)
    slot = eng.new_sequence()
    eng.cache.reserve(slot, len(toks))
    eng.cache.upload_tables()
    meta = build_meta([SeqChunk(slot, 0, len(toks), 0)], np.asarray(toks, dtype=np.int32), np.arange(len(toks), dtype=np.int32),
                      eng.ops.device)
    ctx = StepContext(eng.ops, meta, eng.cache)
    ctx.layer_outputs = []
    eng.model.forward(ctx)
    want = []
    plain.forward(cfg, tensors, toks, torch.float64, want)
    assert len(ctx.layer_outputs) == len(want) == 4
    for got, ref in zip(ctx.layer_outputs, want):
        assert cases.rel_err(got, ref) <= TOL


def test_sizes_that_a_tensor_gives_and_tensors_a_layer_does_not_use(tmp_path):
    """config.json may leave out the sizes that a tensor's shape gives; what nothing gives is an error.  A layer without
    feed-forward may still carry its norms."""
    cfg = CONFIGS["A"]
    tensors = make_tensors(cfg, 4)
    bare = json.loads(json.dumps(cfg))
    for layer in bare["layers"]:
        for k in {"attention": ("dim", "vdim", "kv_heads"), "latent_attention": ("dim", "vdim", "kv_rank"),
                  "mamba2": ("heads", "vdim", "state", "conv")}[layer["type"]]:
            layer["mixer"].pop(k)
    bare["layers"][0]["mlp"].pop("ff")
    bare["layers"][1]["mlp"].pop("expert")
    bare["layers"][1]["mlp"]["router"].pop("experts")
    bare["layers"][1]["mlp"]["shared"].pop("ff")
    extra = dict(tensors, **{"l2.norm2": torch.ones(64), "l2.norm2b": torch.zeros(64)})
    toks = tokens_for(cfg, 30, 2)
    eng = Engine.load_path(write_model(tmp_path / "m", bare, extra), dtype="float32", ops=TorchOps(torch.float32),
                           max_tokens=256, verbose=False)
    assert cases.rel_err(cases.run_cut(eng, toks, [7]), plain.forward(cfg, tensors, toks)) <= TOL
    with pytest.raises(ConfigError):
        spec_of(bare)
    with pytest.raises(Exception):
        Engine.load_path(write_model(tmp_path / "n", cfg, dict(tensors, other=torch.zeros(3))), dtype="float32",
                         ops=TorchOps(torch.float32), max_tokens=256, verbose=False)


def test_config_is_read_and_checked(tmp_path):
    cfg = CONFIGS["A"]
    folder = write_model(tmp_path / "m", cfg, make_tensors(cfg, 1))
    assert load_config(folder).residual_mult == 0.4
    assert config_from_dict(load_config(folder).to_dict()) == load_config(folder)
    shapes = spec_of(cfg).expected_shapes()
    assert shapes["embed.norm"] == shapes["final.norm"] == shapes["l0.norm1b"] == shapes["l1.norm2b"] == (64,)
    assert shapes["l0.mix.q"] == (96, 64) and shapes["l0.mix.q.b"] == (96,) and shapes["l0.mix.k.b"] == (48,)
    assert shapes["l0.mix.o.b"] == (64,) and "l0.mix.v" not in shapes and "l0.mix.v.b" not in shapes
    assert shapes["l1.mix.in"] == (2 * 64 + 2 * 2 * 8 + 4, 64) and shapes["l1.mix.conv"] == (64 + 32, 4)
    assert shapes["l1.mix.conv.b"] == (96,) and shapes["l1.mix.norm"] == (64,) and shapes["l1.mix.A_log"] == (4,)
    assert shapes["l1.mlp.router"] == (6, 64) and shapes["l1.mlp.correction"] == (6,) and "l1.mlp.shared.sg" not in shapes
    assert shapes["l2.mix.dkv"] == (40, 64) and shapes["l2.mix.g"] == (3, 64) and "l2.norm2" not in shapes
    assert shapes["l2.mix.uk"] == (48, 40) and shapes["l2.mix.uv"] == (72, 40) and shapes["head"] == (96, 64)
    for path, value in ((("layers", 1, "type"), "other"), (("layers", 0, "mixer", "kv_heads"), 3), (("norm", "eps"), 0),
                        (("layers", 0, "mixer", "vdim"), 12), (("layers", 0, "mixer", "rot", "dims"), 7),
                        (("layers", 0, "mixer", "rot", "scaling"), {"factor": 2.0}), (("layers", 0, "mlp", "kind"), "other"),
                        (("layers", 0, "mixer", "mask"), {"keep_first": 2}), (("layers", 0, "mixer", "mask", "keep_first"), -1),
                        (("layers", 1, "mixer", "groups"), 3), (("layers", 1, "mixer", "norm_groups"), 7),
                        (("layers", 1, "mixer", "conv"), 0), (("layers", 2, "mixer", "mask", "size"), 0),
                        (("layers", 1, "mlp", "router", "top"), 7), (("layers", 1, "mlp", "shared", "ff"), 0),
                        (("residual_mult",), None)):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_engine_from_a_model_folder_and_trace_replay(tmp_path):
    """The folder's config.json chooses the model class; trace replay drives the same engine."""
    from rbitnet_b200 import replay
    import io
    import numpy as np
    cfg = CONFIGS["A"]
    tensors = make_tensors(cfg, 5)
    folder = write_model(tmp_path / "m", cfg, tensors, store=torch.bfloat16)
    a, b = tokens_for(cfg, 9, 1), tokens_for(cfg, 4, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:6], "want": [0, 5]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[6:7], "want": []}, {"id": "b", "tokens": b[3:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[7:], "want": [1]}], "end": ["a"]}]
    out = io.StringIO()
    rc = replay.main(["--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "64"],
                     stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), stdout=out, ops=TorchOps(torch.float32))
    assert rc == 0 and out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    ra, rb = plain.forward(cfg, tensors, a), plain.forward(cfg, tensors, b)
    got = [torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4").reshape(n, -1)) for i, n in enumerate((3, 1, 1))]
    assert cases.rel_err(got[0], torch.stack([ra[0], ra[5], rb[2]])) <= TOL
    assert cases.rel_err(got[1], rb[3:4]) <= TOL and cases.rel_err(got[2], ra[8:9]) <= TOL
