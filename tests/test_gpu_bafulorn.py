"""The Bafulorn decoder on the GPU: the package's kernels against the plain implementation (whole models in both
dtypes, the same cases as on the CPU), and each new kernel alone against the plain functions."""
import numpy as np
import pytest
import torch

import plain_bafulorn as plain
import bafulorn_cases as cases
from safuvik_tiny import tokens_for, rel_err, run_cut
from bafulorn_tiny import CONFIGS, make_tensors, model, latent_layer, attention_layer, mamba_layer, dense, moe
from rbitnet_b200.config import config_from_dict

pytestmark = pytest.mark.gpu

# Fractions of the largest reference value.  float32: the weights are scaled up so that faults show, which amplifies
# rounding.  bfloat16: operands of the products, the convolved channels, q, the cache, the attention's P and the rows between a
# feed-forward's products are rounded to 8 bits; there the matrices are spread less, and a router's choice may fall the other
# way where two scores are closer than the rounding of its input rows (single positions, see ``Band``).
TOL = {"float32": 2e-4, "bfloat16": 6e-2}
BAND = {"float32": cases.Band(2e-4), "bfloat16": cases.Band(6e-2, spikes=0.1, spread=5.0)}
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def engine_maker(dtype):
    from rbitnet_b200.engine import Engine

    def make(cfg, tensors, max_tokens=64 * 16, graphs=False, **kw):
        return Engine(config_from_dict(cfg), dict(tensors), dtype=dtype, max_tokens=max_tokens, max_seq=1024,
                      use_graphs=graphs, **kw)
    return make


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole(name, dtype):
    cases.whole(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_prefill_against_decoding(name, dtype):
    cases.prefill_against_decoding(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", list(range(101, 121)))
def test_random_configurations(seed, dtype):
    cases.random_configuration(engine_maker(dtype), seed, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions(name, dtype):
    cases.portions(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_batches(name, dtype):
    cases.batches_against_alone(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_slots_and_pages_used_again(name, dtype):
    cases.slots_and_pages_used_again(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_long_decoding(name, dtype):
    cases.long_decoding(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_first_tokens(name, dtype):
    cases.first_tokens(engine_maker(dtype), name, BAND[dtype])


def _cuts(n):
    return ([], [n - 40, n - 2, n - 1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_rank", [16, 64, 128, 192])
@pytest.mark.parametrize("n,far,window,keep,seen", cases.KEYS)
def test_one_key_of_the_latent_attention(n, far, window, keep, seen, kv_rank, dtype):
    for cuts in _cuts(n):
        cases.one_key_stands_out(engine_maker(dtype), TOL[dtype], "latent", n, far, window, keep, seen, cuts,
                                 last_only=dtype == "bfloat16", kv_rank=kv_rank)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("n,far,window,keep,seen", cases.KEYS + cases.KEPT_KEYS)
def test_one_key_of_the_attention(n, far, window, keep, seen, dim, dtype):
    for cuts in _cuts(n):
        cases.one_key_stands_out(engine_maker(dtype), TOL[dtype], "attention", n, far, window, keep, seen, cuts,
                                 last_only=dtype == "bfloat16", dim=dim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[], [2, 100, 101, 250], [390] + list(range(391, 400))])
def test_state_carries_the_first_token(cuts, dtype):
    cases.state_carries_the_first_token(engine_maker(dtype), TOL[dtype] / 2, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[], [40, 63, 64, 100], list(range(1, 150))])
def test_turned_part(cuts, dtype):
    cases.turned_part_decides(engine_maker(dtype), TOL[dtype], cuts, last=None if dtype == "float32" else 100)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_greedy_generation_through_captured_steps(name):
    cases.greedy_generation(engine_maker("float32"), name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_captured_step(name, dtype):
    """The captured decode step (the trial run before the capture must leave the states as they were; padding rows) against
    the plain model."""
    from rbitnet_b200.engine.step import StepEntry
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, 23, spread=BAND[dtype].spread)
    eng = engine_maker(dtype)(cfg, tensors, graphs=True)
    reqs = [tokens_for(cfg, n, 70 + n) for n in (90, 9, 163)]
    slots = [eng.new_sequence() for _ in reqs]
    eng.step([StepEntry(s, r[:-6], []) for s, r in zip(slots, reqs)])
    got = [[] for _ in reqs]
    for k in range(6, 0, -1):
        out = eng.step([StepEntry(s, [r[-k]], [0]) for s, r in zip(slots, reqs)], captured=True)
        for i in range(len(reqs)):
            got[i].append(out[i:i + 1])
    assert BAND[dtype].ok_all([(torch.cat(got[i]).float().cpu(), plain.forward(cfg, tensors, r)[-6:]) for i, r in enumerate(reqs)])


def _mid_sizes():
    """Sizes that every tensor-core kernel takes, products whose K is cut into clusters, cached rows of 128 and heads of 128."""
    return model(1000, 768, [
        mamba_layer(16, 64, 128, 4, 4, 4, dense(1024)),
        latent_layer(12, 64, 64, 128, 90, 0.12, moe(24, 4, 256, shared=512, scale=2.5)),
        attention_layer(8, 2, 128, 100, 70, 0.09, 128, moe(24, 4, 256, shared=512, scale=2.5), base=1e5, scaling=(4.0, 1.0, 4.0, 128)),
        mamba_layer(24, 32, 64, 1, 4, 1, None)], mult=0.4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mid_sizes(dtype):
    """Whole, the last 40 tokens one by one, and an unequal batch decoded together, at sizes of the tensor-core kernels."""
    from rbitnet_b200.engine.step import StepEntry
    cfg = _mid_sizes()
    band = BAND[dtype]
    tensors = make_tensors(cfg, seed=31, spread=band.spread)
    eng = engine_maker(dtype)(cfg, tensors, max_tokens=64 * 16)
    toks = tokens_for(cfg, 300, 9)
    ref = plain.forward(cfg, tensors, toks)
    assert band.ok(run_cut(eng, toks, []), ref)
    assert band.ok(run_cut(eng, toks, list(range(260, 300))), ref)
    reqs = [toks[:150], tokens_for(cfg, 70, 10), tokens_for(cfg, 9, 11)]
    refs = [ref[:150]] + [plain.forward(cfg, tensors, r) for r in reqs[1:]]
    slots = [eng.new_sequence() for _ in reqs]
    cut = [len(r) - 5 for r in reqs]
    out = eng.step([StepEntry(s, r[:n], list(range(n))) for s, r, n in zip(slots, reqs, cut)])
    got, at = [], 0
    for n in cut:
        got.append([out[at:at + n]])
        at += n
    for k in range(5):
        out = eng.step([StepEntry(s, [r[n + k]], [0]) for s, r, n in zip(slots, reqs, cut)])
        for i in range(len(reqs)):
            got[i].append(out[i:i + 1])
    assert band.ok_all([(torch.cat(g).float().cpu(), r) for g, r in zip(got, refs)])


def test_command_line_and_trace_replay(tmp_path):
    """``python -m rbitnet_b200 random`` makes a model of the design from its config.json; ``generate --temperature 0``
    prints the plain model's greedy ids; ``bin/trace_run`` replays a schedule of two unequal requests on the same folder."""
    import json
    import os
    import subprocess
    import sys
    from pathlib import Path
    from rbitnet_b200.weights import read_safetensors
    root = Path(__file__).resolve().parent.parent
    cfg = CONFIGS["D"]
    (tmp_path / "cfg.json").write_text(json.dumps(cfg))
    env = dict(os.environ, PYTHONPATH=str(root))
    folder = tmp_path / "model"
    p = subprocess.run([sys.executable, "-m", "rbitnet_b200", "random", "--config", str(tmp_path / "cfg.json"), "--out", str(folder),
                        "--seed", "5", "--dtype", "float32"], capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    tensors = {k: v.float() for k, v in read_safetensors(folder / "model.safetensors").items()}
    ps = [tokens_for(cfg, 7, 1), tokens_for(cfg, 3, 2)]
    cmd = [sys.executable, "-m", "rbitnet_b200", "generate", "--model", str(folder), "--dtype", "float32", "--temperature", "0",
           "--max-tokens", "6", "--cache-tokens", "512"]
    for q in ps:
        cmd += ["--prompt-ids", " ".join(map(str, q))]
    p = subprocess.run(cmd, capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [json.loads(x) for x in p.stdout.strip().splitlines()]
    assert len(lines) == 2
    for q, rec in zip(ps, lines):
        seq = list(q)
        for tok in rec["tokens"]:
            logits = plain.forward(cfg, tensors, seq)[-1]
            best = int(torch.argmax(logits))
            assert best == tok or float(logits[best] - logits[tok]) <= 1e-4 * float(logits.abs().max())
            seq.append(tok)
        assert len(rec["tokens"]) == 6
    a, b = tokens_for(cfg, 70, 3), tokens_for(cfg, 5, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 64, 65]}, {"id": "b", "tokens": b[:4], "want": [3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[4:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[67:68], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:], "want": [0, 1]}], "end": ["a"]}]
    ra, rb = plain.forward(cfg, tensors, a), plain.forward(cfg, tensors, b)
    want = {0: torch.stack([ra[0], ra[64], ra[65], rb[3]]), 1: torch.stack([ra[66], rb[4]]), 3: torch.stack([ra[68], ra[69]])}
    for dtype in DTYPES:
        out = tmp_path / f"out_{dtype}"
        p = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128"], input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True,
                           text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert p.stdout.split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
        assert not (out / "2.f32").exists()
        for i, ref in want.items():
            got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(ref.shape[0], -1))
            assert rel_err(got, ref) <= TOL[dtype], (dtype, i)


# ---------------------------------------------------------------- kernels alone
def _ops(dtype):
    from rbitnet_b200.kernels.ops import CudaOps
    return CudaOps(TORCH.get(dtype, dtype))


def _meta(ops, runs):
    """runs: (slot, start, n) per sequence."""
    from rbitnet_b200.engine.step import SeqChunk, build_meta
    chunks, at = [], 0
    for slot, start, n in runs:
        chunks.append(SeqChunk(slot, start, n, at))
        at += n
    return build_meta(chunks, np.zeros(at, dtype=np.int32), np.zeros(0, dtype=np.int32), ops.device)


class _Ctx:
    def __init__(self, ops, meta=None, cache=None, state=None):
        self.ops, self.meta, self._cache, self._state = ops, meta, cache, state

    def cache_view(self, entry):
        return self._cache.view(0)

    def state_view(self, entry):
        return self._state


def _rounded(g, *shape, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).double()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fresh", [False, True])
@pytest.mark.parametrize("T,E", [(1, 64), (7, 100), (300, 1024), (3, 4104), (5, 7), (600, 2048), (9, 8192), (2, 18432), (40, 2052)])
def test_a_results_norm_and_the_norm_after_it(dtype, fresh, T, E):
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(E)
    x, y = torch.randn(T, E, generator=g, dtype=torch.float64), torch.randn(T, E, generator=g, dtype=torch.float64) * 30.0
    y[0] *= 1e-4                                                       # eps matters
    w, w2 = torch.randn(E, generator=g, dtype=torch.float64), torch.randn(E, generator=g, dtype=torch.float64)
    xd = None if fresh else x.float().cuda()
    got, h = ops.norm_add_norm(xd, y.float().cuda(), w.float().cuda(), 1e-5, w2.float().cuda(), 1e-3)
    want = (0.0 if fresh else x) + plain.rms(y, 1e-5) * w
    assert fresh or got.data_ptr() == xd.data_ptr()
    assert rel_err(got.cpu(), want) <= 2e-6 and h.dtype == TORCH[dtype]
    assert rel_err(h.float().cpu(), plain.rms(want, 1e-3) * w2) <= (3e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,groups", [(3, 64, 2), (300, 4096, 8), (8, 4096, 1), (5, 1024, 4), (2, 2048, 1), (7, 1028, 1), (4, 300, 1),
                                        (6, 8200, 2), (3, 777, 3)])
def test_norm_in_equal_parts(dtype, T, E, groups):
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(E)
    x, w = torch.randn(T, E, generator=g, dtype=torch.float64), torch.randn(E, generator=g, dtype=torch.float64)
    x[:, :E // groups] *= 1e-2
    got = ops.rmsnorm_grouped(x.float().cuda(), w.float().cuda(), groups, 1e-5)
    want = plain.rms(x.view(T, groups, -1), 1e-5).reshape(T, E) * w
    assert rel_err(got.float().cpu(), want) <= (2e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("H,Kh,D,shared", [(4, 2, 64, False), (8, 8, 128, False), (8, 2, 48, False), (6, 1, 80, False), (3, 1, 40, False),
                                           (5, 1, 64, True), (16, 1, 128, True), (20, 1, 128, True), (4, 1, 192, True), (16, 1, 256, True)])
@pytest.mark.parametrize("window,keep", [(100, 23), (64, 64), (33, 70), (130, 200), (5, 1), (1, 3), (300, 129)])
def test_attention_with_kept_first_positions(H, Kh, D, shared, window, keep):
    """Every attention kernel (prompts on tensor memory and on mma.sync, decode steps by TMA, by cp.async and in parts, the
    plain one) in both dtypes against the plain function: prompts that begin anywhere, decode steps over short and long
    contexts, the keys behind the window and the kept positions filled with large values."""
    import dataclasses
    from rbitnet_b200.cache import SequenceCache
    from rbitnet_b200.parts.base import CacheNeed
    runs = {"decode": [(700, 1), (70, 1), (1, 1), (129, 1)], "one decode": [(900, 1)],
            "prompts": [(300, 300), (400, 37), (64, 64), (193, 2), (128, 1)], "long prompt": [(700, 500)]}
    for dtype in (torch.float32, torch.bfloat16):
        ops = _ops(dtype)
        for what, seqs in runs.items():
            need = CacheNeed(Kh, D, None, streams=((Kh, D),) if shared else None)
            cache = SequenceCache({0: need}, {}, {}, 64 * 40, 1024, dtype, ops.device)
            slots = [cache.alloc() for _ in seqs]
            for s, (n, _) in zip(slots, seqs):
                cache.reserve(s, n)
            cache.upload_tables()
            view = cache.view(0)
            view = dataclasses.replace(view, v=view.k) if shared else view
            gen = torch.Generator().manual_seed(D + H)
            k, v = _rounded(gen, *view.k.shape, scale=0.7), _rounded(gen, *view.k.shape, scale=0.7)
            view.k.copy_(k.to(dtype))
            if shared:
                v = k
            else:
                view.v.copy_(v.to(dtype))
            T = sum(m for _, m in seqs)
            q = _rounded(gen, T, H, D, scale=0.7)
            scale = 1.5 * D ** -0.5
            meta = _meta(ops, [(s, n - m, m) for s, (n, m) in zip(slots, seqs)])
            got = ops.attention(q.to(dtype).cuda(), meta, view, H, scale, window, keep_first=keep).float().cpu()
            table = view.page_table.cpu().long()
            at, want = 0, []
            for s, (n, m) in zip(slots, seqs):
                idx = torch.arange(n)
                ks, vs = k[table[s, idx // 64], :, idx % 64], v[table[s, idx // 64], :, idx % 64]
                full = torch.zeros(n, H, D, dtype=torch.float64)
                full[n - m:] = q[at:at + m]
                see = plain.visible(n, {"size": window, "keep_first": keep})
                want.append(plain.softmax_attention(full, ks, vs, scale, see)[n - m:].reshape(m, H * D))
                at += m
            assert rel_err(got, torch.cat(want)) <= (2e-5 if dtype == torch.float32 else 1.5e-2), (what, dtype)
        ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,N,K,stride", [(1, 3, 8, 16, 16), (8, 16, 128, 96, 128), (16, 2, 33, 100, 112), (17, 2, 33, 100, 112),
                                            (300, 3, 40, 24, 24), (300, 5, 128, 96, 128), (513, 2, 256, 128, 160), (260, 6, 200, 64, 64)])
def test_a_matrix_per_head_with_a_gate_per_head(dtype, T, H, N, K, stride):
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(T * 10 + H)
    x, w = _rounded(g, T, H * stride), _rounded(g, H, N, K, scale=0.3)
    rows = torch.randn(T, 7 + H, generator=g, dtype=torch.float64) * 2.0
    weight = ops.prepare_per_head(w.float().cuda())
    want = torch.einsum("thk,hnk->thn", x.view(T, H, stride)[..., :K], w) * torch.sigmoid(rows[:, 7:])[:, :, None]
    for on in (True, False):
        ops.per_head_on_tensor_cores = on
        got = ops.per_head_linear(x.to(TORCH[dtype]).cuda(), weight, gate=(rows.float().cuda(), 7, "head"))
        assert rel_err(got.float().cpu(), want.reshape(T, H * N)) <= (1e-5 if dtype == "float32" else 1e-2), on
    # the gate per head is of the one call only
    per_value = torch.randn(T, H * N, generator=g, dtype=torch.float64)
    got = ops.per_head_linear(x.to(TORCH[dtype]).cuda(), weight, gate=(per_value.float().cuda(), 0))
    want = torch.einsum("thk,hnk->thn", x.view(T, H, stride)[..., :K], w).reshape(T, H * N) * torch.sigmoid(per_value)
    assert rel_err(got.float().cpu(), want) <= (1e-5 if dtype == "float32" else 1e-2)
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("T,E,F", [(1, 256, 96), (8, 64, 40), (16, 128, 24), (130, 64, 200), (700, 128, 1024), (9, 50, 30)])
def test_gated_feed_forward_with_relu(dtype, fused, T, E, F):
    from rbitnet_b200.parts.feed_forward import GatedDense
    ops = _ops(dtype)
    ops.fuse_gated_act = fused
    g = torch.Generator().manual_seed(T + F)
    part = GatedDense(E, F, "relu")
    w = {k: _rounded(g, *s, scale=1.2 * s[-1] ** -0.5) for k, (s, _) in part.weight_shapes().items()}
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    got = part.forward(_Ctx(ops), h.to(TORCH[dtype]).cuda()).cpu()
    assert rel_err(got, plain.gated_ff(h, w["gate"], w["up"], w["down"], plain.relu)) <= (1e-5 if dtype == "float32" else 1e-2)
    ops.check_errors()


@pytest.mark.parametrize("n,top,T,K,scale", [(16, 1, 50, 48, 2.0), (5, 2, 333, 100, 1.0), (3, 3, 7, 70, 0.5), (60, 6, 200, 64, 2.5),
                                             (2, 1, 1, 32, 3.0), (70, 40, 9, 64, 1.5), (14, 5, 8, 264, 1.25)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_router_with_divided_weights(dtype, n, top, T, K, scale):
    """Sigmoid scores, a correction that only decides the choice, the chosen scores divided by their sum and scaled; on the
    tensor cores, from a product's sums and in one kernel."""
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(n * 10 + top)
    h, router, corr = _rounded(g, T, K), _rounded(g, n, K, scale=3.0 * K ** -0.5), _rounded(g, n, scale=0.3)
    for tc in {None, ops.prepare_router(router.float().cuda())} if dtype == "float32" else (None, ops.prepare_router(router.float().cuda())):
        ids, weights, _ = ops.route_scored(h.to(TORCH[dtype]).cuda(), router.float().cuda(), corr.float().cuda(), top, 0, 0,
                                           scoring="sigmoid", router_tc=tc, normalize=1e-20, weight_scale=scale)
        z = h @ router.T
        ids, weights = ids.cpu().long(), weights.cpu().double()
        for t in range(T):
            want_ids, want = plain.choose(z[t], corr, top, scale)
            assert ids[t].tolist() == want_ids.tolist(), t
            assert float((weights[t] - want).abs().max()) <= 1e-5 * scale
    # the weighing is of one call only
    _, weights, _ = ops.route_scored(h.to(TORCH[dtype]).cuda(), router.float().cuda(), None, top, 0, 0, scoring="sigmoid")
    want = torch.sigmoid(h @ router.T).sort(-1, descending=True).values[:, :top]
    assert float((weights.cpu().double() - want).abs().max()) <= 1e-5
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,F,n,top,shared", [(1, 64, 40, 6, 2, 48), (3, 64, 40, 6, 6, None), (70, 64, 24, 3, 1, 24),
                                                (300, 128, 72, 16, 4, 256), (45, 100, 36, 4, 2, 20), (9, 50, 30, 2, 1, 10)])
def test_experts_with_a_shared_one_without_a_gate(dtype, T, E, F, n, top, shared):
    from rbitnet_b200.parts.feed_forward import RoutedExperts
    ops = _ops(dtype)
    g = torch.Generator().manual_seed(T + E)
    part = RoutedExperts(E, F, n, top, activation="silu", scoring="sigmoid", normalize=1e-20, weight_scale=2.0,
                         shared={"inner": shared, "gate": False} if shared else None)
    w = {k: _rounded(g, *s, scale=(1.5 * s[-1] ** -0.5 if len(s) > 1 else 0.2)) for k, (s, _) in part.weight_shapes().items()}
    assert "shared.sg" not in w
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    mlp = {"router": {"experts": n, "top": top, "scale": 2.0}}
    if shared:
        mlp["shared"] = {"ff": shared}
    want = plain.routed_ff(h, mlp, w)
    assert rel_err(part.forward(_Ctx(ops), h.to(TORCH[dtype]).cuda()).cpu(), want) <= (1e-5 if dtype == "float32" else 2e-2)
    x0 = torch.randn(T, E, generator=g, dtype=torch.float64)
    x = x0.float().cuda()
    part.forward(_Ctx(ops), h.to(TORCH[dtype]).cuda(), accumulate_into=x)
    assert rel_err(x.cpu() - x0, want) <= (2e-5 if dtype == "float32" else 2e-2)
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("what,args", [
    ("latent", (4, 16, 24, 40, 50)), ("latent", (16, 64, 64, 128, 33)), ("latent", (3, 10, 7, 13, 70)), ("latent", (2, 32, 128, 64, None)),
    ("attention", (4, 2, 64, 40, 5, 64)), ("attention", (8, 2, 128, 30, 66, 64)), ("attention", (3, 3, 10, 17, 3, 4)),
    ("attention", (4, 1, 48, None, 0, 0))])
def test_attention_parts(dtype, what, args):
    """The two attention mixers over the paged cache: whole, in portions across a page border, and token by token."""
    from rbitnet_b200.cache import SequenceCache
    from rbitnet_b200.parts.latent import LatentAttention
    from rbitnet_b200.parts.attention import Attention
    ops = _ops(dtype)
    E, T, g = 64, 150, torch.Generator().manual_seed(sum(a or 0 for a in args))
    if what == "latent":
        H, D, Dv, C, window = args
        part = LatentAttention(E, H, D, Dv, 0, C, scale=D ** -0.5, norm_eps=1e-5, window=window, head_gate=True)
        m = latent_layer(H, D, Dv, C, window, D ** -0.5)["mixer"]
    else:
        H, Kh, D, window, keep, rot = args
        pos = {"kind": "rotary", "params": {"head_dim": D, "theta": 50.0, "pairing": "half", "rot_dim": rot}} if rot else None
        part = Attention(E, H, Kh, D, position=pos, window=window, keep_first=keep, scale=D ** -0.5, values="keys", bias=True)
        m = attention_layer(H, Kh, D, window, keep, D ** -0.5, rot, base=50.0)["mixer"]
    w = {k: _rounded(g, *s, scale=1.2 * s[-1] ** -0.5 if len(s) > 1 else 0.5) for k, (s, _) in part.weight_shapes().items()}
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    want = plain.latent_attention(h, m, w, 1e-5) if what == "latent" else plain.attention(h, m, w)
    for cuts in ([0, T], [0, 1, 2, 63, 64, 66, 130, T], list(range(T + 1))):
        cache = SequenceCache({0: part.cache_need()}, {}, {}, 64 * 4, 256, TORCH[dtype], ops.device)
        cache.alloc()
        slot = cache.alloc()
        outs = []
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            cache.reserve(slot, hi - lo)
            cache.upload_tables()
            ctx = _Ctx(ops, _meta(ops, [(slot, lo, hi - lo)]), cache=cache)
            outs.append(part.forward(ctx, h[lo:hi].to(TORCH[dtype]).cuda(), 0))
            cache.advance(slot, hi - lo)
        assert rel_err(torch.cat(outs).cpu(), want) <= (2e-5 if dtype == "float32" else 3e-2), cuts
    ops.check_errors()


#: heads, value_dim, state rows, groups, taps
SSD = [(2, 16, 32, 1, 4), (8, 64, 128, 2, 4), (3, 7, 5, 3, 5), (4, 80, 64, 4, 2), (2, 128, 256, 1, 3), (6, 24, 20, 2, 1), (1, 33, 130, 1, 4),
       (4, 8, 400, 1, 4)]


def _ssd(ops, H, P, N, G, K, seed=0, forget=0.0):
    from rbitnet_b200.parts.ssd import StateSpace
    g = torch.Generator().manual_seed(seed + H * 100 + P)
    part = StateSpace(48, H, P, N, G, K, 1, 1e-5)
    w = {k: _rounded(g, *s, scale=0.5) for k, (s, _) in part.weight_shapes().items()}
    w["A_log"] = torch.linspace(-5.0, 1.0, H).double() + forget
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    return part, w, g


def _plain_v(proj, w, H, P, N, G):
    """What ``state_space`` returns for the rows of one whole sequence."""
    T, inner = proj.shape[0], H * P
    u = plain.silu(plain.causal_convolution(proj[:, inner:2 * inner + 2 * G * N], w["conv"], w["conv.b"]))
    y = plain.state_space(u[:, :inner].reshape(T, H, P), u[:, inner:inner + G * N].reshape(T, G, N), u[:, inner + G * N:].reshape(T, G, N),
                          plain.softplus(proj[:, 2 * inner + 2 * G * N:2 * inner + 2 * G * N + H] + w["dt_bias"]), w["A_log"], w["D"])
    return y.reshape(T, inner) * plain.silu(proj[:, :inner])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,P,N,G,K", SSD)
def test_state_space_runs_steps_and_slots(dtype, H, P, N, G, K):
    """Three sequences whose rows come in steps of unequal runs, token by token, and mixed, through the kernels of the state
    space; slots of their own, the state and the convolution's inputs carried from step to step."""
    ops = _ops(dtype)
    part, w, g = _ssd(ops, H, P, N, G, K)
    width = part.w_in.n_out
    lengths, slots = (150, 7, 66), (3, 0, 2)
    proj = [torch.randn(n, width, generator=g, dtype=torch.float64).float().double() for n in lengths]
    want = [_plain_v(x, w, H, P, N, G) for x in proj]
    tol = 3e-5 if dtype == "float32" else 2e-2
    for cuts in ([[0, 150], [0, 7], [0, 66]], [[0, 2, 64, 65, 129, 150], [0, 3, 4, 5, 6, 7], [0, 1, 33, 64, 65, 66]],
                 [list(range(151)), list(range(8)), list(range(67))]):
        state = {"S": torch.zeros(4, H, N, P, device="cuda"), "tail": torch.zeros(4, K, part.channels, device="cuda")}
        got = [[], [], []]
        for step in range(max(len(c) for c in cuts) - 1):
            live = [i for i in range(3) if step + 1 < len(cuts[i])]
            meta = _meta(ops, [(slots[i], cuts[i][step], cuts[i][step + 1] - cuts[i][step]) for i in live])
            rows = torch.cat([proj[i][cuts[i][step]:cuts[i][step + 1]] for i in live]).float().cuda()
            out, at = ops.state_space(rows, part, state, meta).cpu(), 0
            for i in live:
                n = cuts[i][step + 1] - cuts[i][step]
                got[i].append(out[at:at + n])
                at += n
        for i in range(3):
            assert rel_err(torch.cat(got[i]), want[i]) <= tol, (cuts[i][:4], i)
        assert float(state["S"][1].abs().max()) == 0.0 and float(state["tail"][1].abs().max()) == 0.0
    ops.check_errors()


@pytest.mark.parametrize("H,P,N,G,K", [s for s in SSD if s[2] <= 256])
@pytest.mark.parametrize("forget", [-3.0, 0.0, 4.0])
def test_chunks_sum_in_float32(H, P, N, G, K, forget):
    """The chunked kernels against the token-by-token form on the same bfloat16 channels: their sums are those of float32
    operands, with states that hardly forget and with ones that forget within a token."""
    ops = _ops("bfloat16")
    part, w, g = _ssd(ops, H, P, N, G, K, forget=forget)
    runs = [(0, 0, 200), (1, 5, 64), (2, 0, 1), (3, 9, 129)]
    meta = _meta(ops, runs)
    rows = torch.randn(meta.n_tokens, part.w_in.n_out, generator=g).cuda()
    S0 = torch.randn(4, H, N, P, generator=g).cuda()
    tail0 = torch.randn(4, K, part.channels, generator=g).cuda()
    results = {}
    for chunks in (True, False):
        ops.ssd_in_chunks = chunks
        state = {"S": S0.clone(), "tail": tail0.clone()}
        before = ops.lib.launches
        out = ops.state_space(rows, part, state, meta)
        results[chunks] = (out.cpu().double(), state["S"].cpu().double(), state["tail"].cpu(), ops.lib.launches - before)
    assert results[True][3] == 4 and torch.equal(results[True][2], results[False][2])
    for i in (0, 1):
        assert rel_err(results[True][i], results[False][i]) <= (8e-6 if forget > 0 else 4e-6), i
    ops.check_errors()
