"""The Busavik decoder through the package's host logic (configuration, parts, cache manager, step function, scheduler,
generation, trace replay) on the CPU stand-in of the kernel layer, against the plain implementation."""
import json

import pytest
import torch

import plain_busavik as plain
import busavik_cases as cases
from safuvik_tiny import write_model, tokens_for
from busavik_tiny import CONFIGS, make_tensors, spec_of, model, latent_layer, moe
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
    cases.whole(make_engine, name, BAND, n=70)


@pytest.mark.parametrize("name", ["A", "B"])
def test_prefill_against_decoding(name):
    cases.prefill_against_decoding(make_engine, name, BAND, n=30, prompt=13)


@pytest.mark.parametrize("seed", [1, 2, 3, 4])
def test_random_configurations(seed):
    cases.random_configuration(make_engine, seed, BAND, n=100)


def test_portions():
    cases.portions(make_engine, "B", BAND, n=132)


def test_batches():
    cases.batches_against_alone(make_engine, "B", BAND, lengths=(1, 2, 67, 9), decode=6)


def test_slots_and_pages_used_again():
    cases.slots_and_pages_used_again(make_engine, "D", BAND)


def test_first_tokens():
    cases.first_tokens(make_engine, "D", BAND)


def test_one_far_key():
    cases.one_far_key_stands_out(make_engine, TOL, n=150, far=3, cuts=[100, 148, 149])


def test_turned_part():
    cases.turned_part_decides(make_engine, TOL, cuts=[40, 63, 64, 100], n=110)


def test_greedy_generation():
    cases.greedy_generation(make_engine, "A", prompts=(5, 1, 12), new=8)


# ---- every mechanism of the plain implementation against an independent statement of it
def test_plain_rotation_and_stretched_frequencies():
    import math
    torch.manual_seed(1)
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    y = plain.rotate(x, {"base": 100.0, "dims": 4})
    for t in range(5):
        for i, f in enumerate((1.0, 0.1)):
            c, s = math.cos(t * f), math.sin(t * f)
            assert torch.allclose(y[t, :, i], x[t, :, i] * c - x[t, :, i + 2] * s)
            assert torch.allclose(y[t, :, i + 2], x[t, :, i + 2] * c + x[t, :, i] * s)
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
    # 8 dims, base e^8: pair i turns by e^(-2 i), and the place of t turns in `original` is (1/2) ln(original / (2 pi t));
    # original = 2 pi e^3, fast = 1 and slow = e^-2 put the ramp's ends at floor(1.5) and ceil(2.5)
    rot = {"base": math.exp(8.0), "dims": 8, "scaling": {"factor": 5.0, "original": 2 * math.pi * math.exp(3.0), "fast": 1.0,
                                                         "slow": math.exp(-2.0)}}
    f, magnitude = plain.turns(rot)
    want = [1.0, math.exp(-2.0), math.exp(-4.0) * (0.5 / 5.0 + 0.5), math.exp(-6.0) / 5.0]
    assert all(abs(a - b) < 1e-12 for a, b in zip(f, want)) and abs(magnitude - (0.1 * math.log(5.0) + 1.0)) < 1e-15
    z = plain.rotate(x[..., :2].repeat(1, 1, 4), rot)
    assert torch.allclose(z[0], x[0, :, :2].repeat(1, 4) * magnitude)


def test_plain_attention_norm_and_feed_forward_pieces():
    torch.manual_seed(0)
    q, k, v = torch.randn(4, 2, 3).double(), torch.randn(4, 2, 3).double(), torch.randn(4, 2, 5).double()
    out = plain.causal_attention(q, k, v, 0.7)
    for t in range(4):
        for h in range(2):
            w = torch.exp(torch.stack([(q[t, h] @ k[j, h]) * 0.7 for j in range(t + 1)]))
            assert torch.allclose(out[t, h], (w[:, None] * v[:t + 1, h]).sum(0) / w.sum())
    z = torch.linspace(-4, 4, 9).double()
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert torch.allclose(plain.silu(z), torch.nn.functional.silu(z))
    ids, weights = plain.choose(torch.tensor([0.5, 3.0, -1.0, 2.0]).double(), 2)
    assert ids.tolist() == [1, 3] and torch.allclose(weights, torch.tensor([1.0, torch.e ** -1.0]).double() / (1 + torch.e ** -1.0))
    assert torch.allclose(plain.tanh_norm(torch.tensor([0.5]), torch.tensor([2.0]), torch.tensor([0.1]), torch.tensor(3.0)),
                          2.0 * torch.tanh(torch.tensor([1.5])) + 0.1)
    assert plain.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]


@pytest.mark.parametrize("what", ["gate", "dq.norm", "dkv.norm", "norm's bias", "norm's slope", "a projection's bias", "gelu",
                                  "softmax over all", "shared gate", "loop"])
def test_leaving_a_mechanism_out_shows(what, monkeypatch):
    """A mistake planted in the plain implementation moves its logits far outside the tolerance, so the tests that compare
    with it would see the same mistake in the package."""
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    tensors = make_tensors(cfg, 4)
    toks = tokens_for(cfg, 40, 2)
    ref = plain.forward(cfg, tensors, toks)
    bent = dict(tensors)
    if what == "gate":
        bent.update({k: v * 0.0 for k, v in tensors.items() if k.endswith("mix.g")})
    elif what in ("dq.norm", "dkv.norm"):
        bent.update({k: torch.ones_like(v) for k, v in tensors.items() if k.endswith(what)})
    elif what == "norm's bias":
        bent.update({k: v * 0.0 for k, v in tensors.items() if k.endswith("norm2.b")})
    elif what == "norm's slope":
        bent.update({k: torch.ones_like(v) for k, v in tensors.items() if k.endswith("norm1.alpha")})
    elif what == "a projection's bias":
        bent["l0.mlp.down.b"] = tensors["l0.mlp.down.b"] * 0.0
    elif what == "gelu":
        monkeypatch.setattr(plain, "gelu_tanh", plain.silu)
    elif what == "softmax over all":
        def over_all(z, top):
            p = torch.softmax(z, dim=-1)
            best, ids = torch.sort(p, descending=True)
            return ids[:top], best[:top]
        monkeypatch.setattr(plain, "choose", over_all)
    elif what == "shared gate":
        bent.update({k: v * 0.0 for k, v in tensors.items() if k.endswith("shared.sg")})
    else:
        cfg["loop"]["times"] = 1
    assert cases.rel_err(plain.forward(cfg, bent, toks), ref) > 20 * TOL


def test_every_run_of_a_looped_layer_has_its_own_cache():
    cfg = CONFIGS["A"]
    eng = make_engine(cfg, make_tensors(cfg, 1))
    caches, _, states = eng.model.cache_plan()
    assert [e.layer for e in eng.spec.schedule] == [0, 1, 2, 1, 2] and set(caches) == {0, 1, 2, 3, 4} and not states
    assert caches[0].streams == ((1, 48),) and caches[1].streams == caches[3].streams == ((1, 24),)


def test_residual_after_every_layer_run():
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
    assert len(ctx.layer_outputs) == len(want) == 5
    for got, ref in zip(ctx.layer_outputs, want):
        assert cases.rel_err(got, ref) <= TOL


def test_sizes_that_a_tensor_gives_and_tensors_a_layer_does_not_use(tmp_path):
    """config.json may leave out the sizes that a tensor's shape gives; what nothing gives is an error.  A layer without
    feed-forward may still carry its second norm."""
    cfg = CONFIGS["A"]
    tensors = make_tensors(cfg, 4)
    bare = json.loads(json.dumps(cfg))
    for layer in bare["layers"]:
        for k in ("q_rank", "kv_rank", "vdim"):
            layer["mixer"].pop(k)
        layer["mixer"]["rot"].pop("dims")
    bare["layers"][0]["mlp"].pop("ff")
    bare["layers"][1]["mlp"].pop("expert")
    bare["layers"][1]["mlp"]["router"].pop("experts")
    bare["layers"][1]["mlp"]["shared"].pop("ff")
    extra = dict(tensors, **{"l2.norm2": torch.ones(64), "l2.norm2.b": torch.zeros(64), "l2.norm2.alpha": torch.tensor(0.5)})
    toks = tokens_for(cfg, 12, 2)
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
    assert load_config(folder).loop == {"start": 1, "stop": 3, "times": 2}
    assert config_from_dict(load_config(folder).to_dict()) == load_config(folder)
    shapes = spec_of(cfg).expected_shapes()
    assert shapes["l0.norm1"] == shapes["l0.norm1.b"] == (64,) and shapes["l0.norm1.alpha"] == ()
    assert shapes["l0.mix.dq"] == (20, 64) and shapes["l0.mix.uq"] == (3 * 24, 20) and shapes["l0.mix.dkv"] == (48, 64)
    assert shapes["l0.mix.uk"] == (48, 40) and shapes["l0.mix.uv"] == shapes["l0.mix.g"][:1] + (40,) and shapes["l0.mix.o"] == (64, 72)
    assert shapes["l0.mlp.gate.b"] == (48,) and shapes["l0.mlp.down.b"] == (64,) and shapes["l1.mlp.e5.down"] == (64, 24)
    assert shapes["l1.mlp.router"] == (6, 64) and shapes["l1.mlp.shared.sg"] == (1, 64) and "l1.mlp.gate.b" not in shapes
    assert "l2.norm2" not in shapes and shapes["final.norm.alpha"] == () and shapes["head"] == (96, 64)
    for path, value in ((("layers", 1, "type"), "other"), (("layers", 0, "mixer", "kv_rank"), 0), (("norm", "eps"), 0),
                        (("layers", 0, "mixer", "rot_dim"), 7), (("layers", 0, "mixer", "rot", "dims"), 4),
                        (("layers", 0, "mixer", "rot", "scaling"), {"factor": 2.0}), (("layers", 0, "mlp", "kind"), "other"),
                        (("layers", 1, "mlp", "router", "top"), 7), (("layers", 1, "mlp", "shared", "ff"), 0),
                        (("loop", "stop"), 4), (("loop", "times"), 0), (("layers", 2, "mixer", "rot", "base"), 0),
                        (("logit_scale",), None)):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_options_of_latent_attention_go_together():
    """Sinks with queries through a latent, a gate with queries straight from the rows, and neither turned part nor gate:
    against a few lines of arithmetic."""
    from rbitnet_b200.parts.latent import LatentAttention
    from rbitnet_b200.cache import SequenceCache
    from rbitnet_b200.engine.step import SeqChunk, build_meta
    import numpy as np
    ops = TorchOps(torch.float32)
    E, H, D, Dv, C, T = 24, 2, 6, 5, 10, 9
    for q_rank, R, gate, sinks in ((7, 4, True, True), (0, 4, True, False), (7, 0, True, False), (7, 0, False, True), (0, 0, True, True)):
        pos = {"kind": "rotary", "params": {"head_dim": R, "theta": 30.0, "pairing": "half", "rot_dim": R}} if R else None
        part = LatentAttention(E, H, D, Dv, q_rank, C, scale=0.4, norm_eps=1e-5, rot_dim=R, position=pos, sinks=sinks, value_gate=gate)
        g = torch.Generator().manual_seed(3)
        w = {k: torch.randn(*s, generator=g) * 0.5 for k, (s, _) in part.weight_shapes().items()}
        part.bind(w, ops)
        h = torch.randn(T, E, generator=g)
        cache = SequenceCache({0: part.cache_need()}, {}, {}, 128, 128, torch.float32, ops.device)
        slot = cache.alloc()
        cache.reserve(slot, T)
        cache.upload_tables()
        meta = build_meta([SeqChunk(slot, 0, T, 0)], np.zeros(T, dtype=np.int32), np.zeros(0, dtype=np.int32), ops.device)
        ctx = type("C", (), {"ops": ops, "meta": meta, "cache_view": lambda self, e: cache.view(0)})()
        got = part.forward(ctx, h, 0)
        d = {k: v.double() for k, v in w.items()}
        x = h.double()
        q = (plain.rms(x @ d["dq"].T, 1e-5) * d["dq.norm"]) @ d["uq"].T if q_rank else x @ d["q"].T
        q = q.view(T, H, D + R)
        down = x @ d["dkv"].T
        c = plain.rms(down[:, :C], 1e-5) * d["dkv.norm"]
        k = (c @ d["uk"].T).view(T, H, D)
        if R:
            rot = {"base": 30.0, "dims": R}
            q = torch.cat([q[..., :D], plain.rotate(q[..., D:], rot)], dim=-1)
            k = torch.cat([k, plain.rotate(down[:, C:].view(T, 1, R), rot).expand(T, H, R)], dim=-1)
        v = (c @ d["uv"].T).view(T, H, Dv)
        o = torch.zeros(T, H, Dv).double()
        for t in range(T):
            for hh in range(H):
                e = torch.exp((k[:t + 1, hh] @ q[t, hh]) * 0.4)
                o[t, hh] = (e[:, None] * v[:t + 1, hh]).sum(0) / (e.sum() + (torch.exp(d["sink"][hh]) if sinks else 0.0))
        o = o.reshape(T, H * Dv)
        if gate:
            o = o * torch.sigmoid(x @ d["g"].T)
        assert cases.rel_err(got, o @ d["o"].T) <= 2e-5, (q_rank, R, gate, sinks)


def test_engine_from_a_model_folder_and_trace_replay(tmp_path):
    """The folder's config.json chooses the model class; trace replay drives the same engine."""
    from rbitnet_b200 import replay
    import io
    import numpy as np
    cfg = CONFIGS["D"]
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
