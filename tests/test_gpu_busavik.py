"""The Busavik decoder on the GPU: the package's kernels against the plain implementation (whole models in both
dtypes, the same cases as on the CPU), and each new kernel alone against the plain functions."""
import numpy as np
import pytest
import torch

import plain_busavik as plain
import busavik_cases as cases
from safuvik_tiny import tokens_for, rel_err, run_cut
from busavik_tiny import CONFIGS, make_tensors, model, latent_layer, dense, moe
from rbitnet_b200.config import config_from_dict

pytestmark = pytest.mark.gpu

# Fractions of the largest reference value.  float32: the weights are scaled up so that faults show, which amplifies
# rounding.  bfloat16: operands of the products, q, the cache, the attention's P and the rows between a feed-forward's
# products are rounded to 8 bits; there the matrices are spread less, and a router's choice may fall the other way where
# two logits are closer than the rounding of its input rows (single positions, see ``Band``).
TOL = {"float32": 2e-4, "bfloat16": 6e-2}
BAND = {"float32": cases.Band(2e-4), "bfloat16": cases.Band(6e-2, spikes=0.1, spread=5.0)}
DTYPES = ["float32", "bfloat16"]


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
@pytest.mark.parametrize("seed", list(range(101, 117)))
def test_random_configurations(seed, dtype):
    cases.random_configuration(engine_maker(dtype), seed, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions(name, dtype):
    cases.portions(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_batches(name, dtype):
    cases.batches_against_alone(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_slots_and_pages_used_again(name, dtype):
    cases.slots_and_pages_used_again(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(name, dtype):
    cases.long_decoding(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_first_tokens(name, dtype):
    cases.first_tokens(engine_maker(dtype), name, BAND[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_rank", [16, 56, 120])
@pytest.mark.parametrize("n,far,cuts", [(300, 2, []), (300, 63, [250] + list(range(290, 300))), (200, 64, list(range(1, 200))),
                                        (700, 0, [64, 128, 699]), (130, 127, [129])])
def test_one_far_key(n, far, cuts, kv_rank, dtype):
    cases.one_far_key_stands_out(engine_maker(dtype), TOL[dtype], n, far, cuts, last_only=dtype == "bfloat16", kv_rank=kv_rank)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[], [40, 63, 64, 100], list(range(1, 150))])
def test_turned_part(cuts, dtype):
    cases.turned_part_decides(engine_maker(dtype), TOL[dtype], cuts, last=None if dtype == "float32" else 100)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_greedy_generation_through_captured_steps(name):
    cases.greedy_generation(engine_maker("float32"), name)


@pytest.mark.parametrize("name", ["A", "C"])
def test_captured_step_in_bfloat16(name):
    """The captured decode step (rows that leave the norm's rows for the next product, padding rows) against the plain
    model."""
    from rbitnet_b200.engine.step import StepEntry
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, 23, spread=5.0)
    eng = engine_maker("bfloat16")(cfg, tensors, graphs=True)
    reqs = [tokens_for(cfg, n, 70 + n) for n in (20, 9, 33)]
    slots = [eng.new_sequence() for _ in reqs]
    eng.step([StepEntry(s, r[:-6], []) for s, r in zip(slots, reqs)])
    got = [[] for _ in reqs]
    for k in range(6, 0, -1):
        out = eng.step([StepEntry(s, [r[-k]], [0]) for s, r in zip(slots, reqs)], captured=True)
        for i in range(len(reqs)):
            got[i].append(out[i:i + 1])
    assert BAND["bfloat16"].ok_all([(torch.cat(got[i]).float().cpu(), plain.forward(cfg, tensors, r)[-6:])
                                    for i, r in enumerate(reqs)])


def _mid_sizes():
    """Sizes that every tensor-core kernel takes, products whose K is cut into clusters (so that they leave the rows of the
    norm after them), cached rows of 128 (tcgen05 prefill, TMA decode)."""
    s = (4.0, 128, 32.0, 1.0)
    return model(1000, 768, [
        latent_layer(12, 64, 64, 64, 192, 64, 0.09, dense(1024), scaling=s),
        latent_layer(6, 128, 32, 128, 256, 96, 0.08, moe(24, 4, 256, shared=512), base=1e5, scaling=s),
        latent_layer(12, 64, 64, 64, 192, 64, 0.09, None)], loop=(0, 2, 2), logit_scale=0.3)


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


@pytest.mark.parametrize("rows", [1, 8, 16])
def test_a_decode_step_with_and_without_the_norms_in_other_kernels(rows):
    """A step whose products and weighted sums leave the rows of the norm after them, against the step with every norm a
    kernel of its own: the residual stream is the same, the logits agree to rounding."""
    from rbitnet_b200.engine.step import StepEntry
    cfg = _mid_sizes()
    tensors = make_tensors(cfg, seed=32, spread=4.0)
    logits = {}
    for fold in (True, False):
        eng = engine_maker("bfloat16")(cfg, tensors, max_tokens=64 * 40)
        eng.ops.fold_norms = fold
        slots = [eng.new_sequence() for _ in range(rows)]
        eng.step([StepEntry(s, tokens_for(cfg, 5 + i, i), []) for i, s in enumerate(slots)])
        before = eng.ops.lib.launches
        logits[fold] = eng.step([StepEntry(s, [3 + i], [0]) for i, s in enumerate(slots)]).float().cpu()
        logits[fold, "n"] = eng.ops.lib.launches - before
    assert logits[True, "n"] < logits[False, "n"]
    assert torch.equal(logits[True], logits[False])


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
    return CudaOps(dtype)


def _meta(ops, runs):
    """runs: (slot, start, n) per sequence."""
    from rbitnet_b200.engine.step import SeqChunk, build_meta
    chunks, at = [], 0
    for slot, start, n in runs:
        chunks.append(SeqChunk(slot, start, n, at))
        at += n
    return build_meta(chunks, np.zeros(at, dtype=np.int32), np.zeros(0, dtype=np.int32), ops.device)


class _Ctx:
    def __init__(self, ops, meta=None, cache=None):
        self.ops, self.meta, self._cache = ops, meta, cache

    def cache_view(self, entry):
        return self._cache.view(0)


def _rounded(g, *shape, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).double()


TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E", [(1, 64), (7, 100), (300, 1024), (3, 4104), (5, 7), (600, 2048)])
def test_tanh_in_place_of_a_norm(dtype, T, E):
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(E)
    x = torch.randn(T, E, generator=g, dtype=torch.float64) * 3.0
    w, b = torch.randn(E, generator=g, dtype=torch.float64), torch.randn(E, generator=g, dtype=torch.float64)
    x[0, :4] = torch.tensor([0.0, 1e-6, 60.0, -60.0])
    got = ops.tanh_norm(x.float().cuda(), w.float().cuda(), b.float().cuda(), 0.7)
    assert got.dtype == TORCH[dtype]
    assert rel_err(got.float().cpu(), plain.tanh_norm(x, w, b, 0.7)) <= (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,N,K", [(1, 256, 2048), (5, 100, 64), (16, 1024, 512), (17, 256, 2048), (70, 33, 40), (300, 384, 128),
                                   (700, 2048, 768), (40, 50, 36), (2100, 1024, 2048)])
def test_product_with_a_bias(dtype, T, N, K):
    """Stored and added products with a bias per output: K whole, cut into a cluster and shared between teams of blocks; the
    added product may leave the rows of a tanh that follows."""
    from rbitnet_b200.kernels.ops import TanhRequest
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(T + N)
    h, W, bias = _rounded(g, T, K), _rounded(g, N, K, scale=K ** -0.5), torch.randn(N, generator=g, dtype=torch.float64) * 3
    x0 = torch.randn(T, N, generator=g, dtype=torch.float64)
    nw, nb = torch.randn(N, generator=g, dtype=torch.float64), torch.randn(N, generator=g, dtype=torch.float64)
    lw = ops.prepare_linear([W.float().cuda()])
    bias_d, hd = bias.float().cuda(), h.to(TORCH[dtype]).cuda()
    want = h @ W.T + bias
    assert rel_err(ops.linear(hd, lw, out_dtype=torch.float32, bias=bias_d, scale=1.0).cpu(), want) <= 1e-5
    assert rel_err(ops.linear(hd, lw, out_dtype=torch.float32, bias=bias_d, scale=0.25).cpu(), 0.25 * (h @ W.T) + bias) <= 1e-5
    for ask in (False, True):
        x = x0.float().cuda()
        request = TanhRequest(nw.float().cuda(), nb.float().cuda(), 0.6) if ask else None
        ops.linear(hd, lw, accumulate_into=x, bias=bias_d, then_norm=request)
        assert rel_err(x.cpu(), x0 + want) <= 1e-5
        if request is not None and request.result is not None:
            rows = ops.tanh_norm(x, request.weight, request.bias, request.alpha)
            assert torch.equal(request.result, rows)
    if dtype == "bfloat16" and T <= 16 and K >= 512:
        assert request.result is not None                       # few rows and K cut into a cluster: the rows were left
    # the bias is of the next product only
    assert rel_err(ops.linear(hd, lw, out_dtype=torch.float32).cpu(), h @ W.T) <= 1e-5
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("T,E,F", [(1, 256, 96), (8, 64, 40), (16, 128, 24), (50, 100, 36), (130, 64, 200), (700, 128, 1024), (9, 50, 30)])
@pytest.mark.parametrize("activation,bias", [("gelu_tanh", True), ("gelu_tanh", False), ("silu", True)])
def test_gated_feed_forward_with_biases(dtype, fused, T, E, F, activation, bias):
    from rbitnet_b200.parts.feed_forward import GatedDense
    ops = _ops(TORCH[dtype])
    ops.fuse_gated_act = fused
    g = torch.Generator().manual_seed(T + F)
    part = GatedDense(E, F, activation, bias=bias)
    w = {k: _rounded(g, *s, scale=1.2 * s[-1] ** -0.5 if len(s) > 1 else 1.5) for k, (s, _) in part.weight_shapes().items()}
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    z = {k: w.get(f"{k}.b", 0.0) for k in ("gate", "up", "down")}
    act = plain.gelu_tanh if activation == "gelu_tanh" else plain.silu
    want = (act(h @ w["gate"].T + z["gate"]) * (h @ w["up"].T + z["up"])) @ w["down"].T + z["down"]
    ctx = _Ctx(ops)
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert rel_err(part.forward(ctx, h.to(TORCH[dtype]).cuda()).cpu(), want) <= tol
    x0 = torch.randn(T, E, generator=g, dtype=torch.float64)
    x = x0.float().cuda()
    part.forward(ctx, h.to(TORCH[dtype]).cuda(), accumulate_into=x)
    assert rel_err(x.cpu() - x0, want) <= tol
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gated", [False, True])
@pytest.mark.parametrize("T,H,N,K,stride", [(1, 3, 8, 16, 16), (8, 16, 128, 96, 128), (16, 2, 33, 100, 112), (17, 2, 33, 100, 112),
                                            (5, 4, 7, 300, 300), (300, 3, 40, 24, 24), (300, 5, 128, 96, 128), (70, 4, 64, 72, 80),
                                            (513, 2, 256, 128, 160), (700, 3, 24, 200, 208), (260, 2, 200, 64, 64)])
def test_a_matrix_per_head_with_strides_and_a_gate(dtype, gated, T, H, N, K, stride):
    """Heads whose inputs are wider than what the matrix reads; outputs of whole and of broken tiles; many rows on the tensor
    cores (where the sizes allow) and on the plain kernel alike."""
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(T * 10 + H)
    x, w = _rounded(g, T, H * stride), _rounded(g, H, N, K, scale=0.3)
    rows = torch.randn(T, 7 + H * N, generator=g, dtype=torch.float64) * 2.0
    weight = ops.prepare_per_head(w.float().cuda())
    want = torch.einsum("thk,hnk->thn", x.view(T, H, stride)[..., :K], w).reshape(T, H * N)
    if gated:
        want = want * torch.sigmoid(rows[:, 7:])
    for on in (True, False):
        ops.per_head_on_tensor_cores = on
        before = ops.lib.raw("rb_gemm_tc_kernels_launched")()
        got = ops.per_head_linear(x.to(TORCH[dtype]).cuda(), weight, gate=(rows.float().cuda(), 7) if gated else None)
        assert rel_err(got.float().cpu(), want) <= (1e-5 if dtype == "float32" else 1e-2), on
        if dtype == "bfloat16" and T > 16 and K % 8 == 0:       # the tensor-core product ran where it was asked for
            assert (ops.lib.raw("rb_gemm_tc_kernels_launched")() > before) == on
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layout", ["half", "interleaved"])
@pytest.mark.parametrize("T,H,D,R,C,width", [(1, 2, 16, 8, 24, 32), (9, 16, 128, 32, 96, 128), (16, 3, 10, 6, 7, 16), (17, 3, 10, 6, 7, 16),
                                             (300, 4, 32, 16, 112, 128), (80, 2, 24, 64, 130, 208), (300, 2, 16, 2, 200, 208),
                                             (270, 2, 8, 0, 24, 32)])
def test_query_heads_into_the_latents_space(dtype, layout, T, H, D, R, C, width):
    from rbitnet_b200.parts.position import RotaryEncoding
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(T + C)
    q, w = _rounded(g, T, H * (D + R)), _rounded(g, H, C, D, scale=0.3)
    table = None
    start = 900
    if R:
        enc = RotaryEncoding(R, 200.0, layout, scaling={"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
        enc.bind({}, ops)
        table = enc.table()
    meta = _meta(ops, [(1, start, T)]) if T > 1 else _meta(ops, [(1, start, 1)])
    got = ops.latent_queries(q.to(TORCH[dtype]).cuda(), ops.prepare_per_head(w.float().cuda()), R, width, table, meta).float().cpu()
    heads = q.view(T, H, D + R)
    want = torch.zeros(T, H, width, dtype=torch.float64)
    want[..., :C] = torch.einsum("thk,hnk->thn", heads[..., :D], w)
    if R:
        qr = heads[..., D:]
        if layout == "interleaved":                            # the same rotation on another order of the values
            qr = torch.cat([qr[..., 0::2], qr[..., 1::2]], dim=-1)
        rot = {"base": 200.0, "dims": R, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
        late = torch.zeros(start + T, H, R, dtype=torch.float64)
        late[start:] = qr
        y = plain.rotate(late, rot)[start:]
        if layout == "interleaved":
            y = torch.stack([y[..., :R // 2], y[..., R // 2:]], dim=-1).flatten(-2)
        want[..., C:C + R] = y
    assert rel_err(got.view(T, H, width), want) <= (2e-5 if dtype == "float32" else 1e-2)
    assert float(got.view(T, H, width)[..., C + R:].abs().max() if width > C + R else 0.0) == 0.0
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,R,Dv,Rq,C,sinks", [(4, 16, 8, 8, 20, 24, False), (2, 24, 4, 40, 48, 12, False), (8, 64, 16, 64, 64, 112, True),
                                                 (4, 32, 32, 128, 96, 96, False), (1, 8, 2, 8, 5, 200, False), (2, 64, 64, 16, 32, 64, False),
                                                 (16, 16, 16, 32, 24, 240, True), (3, 10, 6, 7, 11, 13, False), (2, 16, 8, 24, 16, 320, False)])
def test_latent_attention_part(dtype, H, D, R, Dv, Rq, C, sinks):
    """Attention through latents with queries from a latent of their own, a shared turned key part and a gate per value, over
    the paged cache: whole, in portions across a page border, and token by token; cache rows of sizes that the tensor-core
    attention kernels take and refuse."""
    from rbitnet_b200.cache import SequenceCache
    from rbitnet_b200.parts.latent import LatentAttention
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(H * 100 + D)
    E, T, scale = 64, 90, (D + R) ** -0.5
    part = LatentAttention(E, H, D, Dv, Rq, C, scale=scale, norm_eps=1e-5, rot_dim=R, value_gate=True, sinks=sinks, position={
        "kind": "rotary", "params": {"head_dim": R, "theta": 50.0, "pairing": "half", "rot_dim": R}})
    w = {k: _rounded(g, *s, scale=1.2 * s[-1] ** -0.5 if len(s) > 1 else 1.0) for k, (s, _) in part.weight_shapes().items()}
    if sinks:
        w["sink"] = torch.full((H,), -40.0).double()           # a sink that weighs nothing: the plain function has none
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": Dv, "kv_rank": C, "scale": scale, "rot": {"base": 50.0, "dims": R}}
    want = plain.latent_attention(h, m, w, 1e-5)
    for cuts in ([0, T], [0, 1, 2, 63, 64, 66, T], list(range(T + 1))):
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


@pytest.mark.parametrize("n,top,T,K", [(16, 1, 50, 48), (5, 2, 333, 100), (3, 3, 7, 70), (60, 6, 200, 64), (2, 1, 1, 32), (70, 40, 9, 64)])
@pytest.mark.parametrize("extra", [0, 1])
@pytest.mark.parametrize("dtype", DTYPES)
def test_router_with_the_softmax_over_the_chosen(dtype, n, top, T, K, extra):
    ops = _ops(TORCH[dtype])
    g = torch.Generator().manual_seed(n * 10 + top)
    h, router = _rounded(g, T, K), _rounded(g, n + extra, K, scale=3.0 * K ** -0.5)
    tc = ops.prepare_router(router.float().cuda())
    ids, weights, gate = ops.route_scored(h.to(TORCH[dtype]).cuda(), router.float().cuda(), None, top, 0, 0,
                                          scoring="softmax_chosen", extra_rows=extra, router_tc=tc)
    z = h @ router[:n].T
    ids, weights = ids.cpu().long(), weights.cpu().double()
    for t in range(T):
        want_ids, want = plain.choose(z[t], top)
        assert ids[t].tolist() == want_ids.tolist(), t
        assert float((weights[t] - want).abs().max()) <= 1e-5
    assert float((weights.sum(-1) - 1.0).abs().max()) <= 1e-5
    if extra:
        assert rel_err(gate.cpu(), h @ router[n:].T) <= 1e-5
    ops.check_errors()


def test_router_logits_far_apart():
    """Logits in the hundreds: a softmax over all outputs would leave nothing of the second choice's weight in float32, the
    softmax over the chosen ones is exact."""
    ops = _ops(torch.float32)
    z = torch.tensor([[300.0, -500.0, 299.0, -200.0], [-900.0, -905.0, -1000.0, -901.0]])
    h = torch.eye(2)
    ids, weights, _ = ops.route_scored(h.cuda(), z.T.contiguous().cuda(), None, 2, 0, 0, scoring="softmax_chosen")
    e = torch.exp(torch.tensor(-1.0))
    assert ids.cpu().tolist() == [[0, 2], [0, 3]]
    assert float((weights.cpu() - torch.tensor([[1.0, float(e)]] * 2) / (1.0 + e)).abs().max()) <= 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,F,n,top,shared", [(1, 64, 40, 6, 2, 48), (3, 64, 40, 6, 6, None), (70, 64, 24, 3, 1, 24),
                                                (300, 128, 72, 16, 4, 256), (45, 100, 36, 4, 2, 20), (2500, 64, 32, 5, 2, None),
                                                (9, 50, 30, 2, 1, 10)])
@pytest.mark.parametrize("fused", [True, False])
def test_experts(dtype, T, E, F, n, top, shared, fused):
    """Few pairs and many, tiles of every size, experts without any token, sizes that the tensor-core products refuse, with
    and without the shared expert; returned, added, and with the rows of the tanh that follows left by the weighted sum."""
    from rbitnet_b200.kernels.ops import TanhRequest
    from rbitnet_b200.parts.feed_forward import RoutedExperts
    if dtype == "float32" and not fused:
        pytest.skip("float32 has the one form")
    ops = _ops(TORCH[dtype])
    ops.fuse_gated_act = fused
    g = torch.Generator().manual_seed(T + E)
    part = RoutedExperts(E, F, n, top, correction=False, activation="silu", scoring="softmax_chosen",
                         shared={"inner": shared} if shared else None)
    w = {k: _rounded(g, *s, scale=1.5 * s[-1] ** -0.5) for k, (s, _) in part.weight_shapes().items()}
    if n > 2:
        w["router"][1] = 0.0
        w["router"][1, 0] = -1.0              # with the first input value large: an expert that nobody chooses
    part.bind({k: v.float().cuda() for k, v in w.items()}, ops)
    h = _rounded(g, T, E)
    h[:, 0] = 6.0
    mlp = {"router": {"experts": n, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    want = plain.routed_ff(h, mlp, w)
    ctx = _Ctx(ops)
    tol = 1e-5 if dtype == "float32" else 2e-2
    assert rel_err(part.forward(ctx, h.to(TORCH[dtype]).cuda()).cpu(), want) <= tol
    x0 = torch.randn(T, E, generator=g, dtype=torch.float64)
    nw, nb = torch.randn(E, generator=g).cuda(), torch.randn(E, generator=g).cuda()
    for ask in (False, True):
        x = x0.float().cuda()
        request = TanhRequest(nw, nb, 0.8) if ask else None
        part.forward(ctx, h.to(TORCH[dtype]).cuda(), accumulate_into=x, then_norm=request)
        assert rel_err(x.cpu() - x0, want) <= tol
        if ask:
            assert torch.equal(request.result, ops.tanh_norm(x, nw, nb, 0.8))
    ops.check_errors()


@pytest.mark.parametrize("H,D", [(8, 64), (16, 128), (32, 128), (3, 192), (32, 192), (32, 256), (128, 256), (20, 112)])
@pytest.mark.parametrize("sinks,window", [(False, None), (True, None), (False, 100)])
def test_attention_over_rows_that_are_keys_and_values(H, D, sinks, window):
    """One key head whose keys and values are the same cached rows: prompts that begin anywhere in a page and a tile of
    keys, and decode steps over short and long contexts (one whose keys are cut into parts of which some have none),
    against the float32 kernel on the same rounded values."""
    import dataclasses
    from rbitnet_b200.cache import SequenceCache
    from rbitnet_b200.parts.base import CacheNeed
    runs = {"decode": [(1500, 1), (70, 1), (1, 1), (129, 1)], "one decode": [(700, 1)],
            "prompts": [(300, 300), (1000, 37), (64, 64), (193, 2), (128, 1)], "long prompt": [(1100, 900)]}
    results = {}
    for dtype in (torch.float32, torch.bfloat16):
        ops = _ops(dtype)
        for what, seqs in runs.items():
            cache = SequenceCache({0: CacheNeed(1, D, None, streams=((1, D),))}, {}, {}, 64 * 60, 2048, dtype, ops.device)
            slots = [cache.alloc() for _ in seqs]
            for s, (n, _) in zip(slots, seqs):
                cache.reserve(s, n)
            cache.upload_tables()
            view = cache.view(0)
            gen = torch.Generator().manual_seed(D + H)
            view.k.copy_((torch.randn(view.k.shape, generator=gen) * 0.7).to(torch.bfloat16).to(dtype))
            T = sum(n for _, n in seqs)
            q = (torch.randn(T, H, D, generator=gen) * 0.7).to(torch.bfloat16).to(dtype).cuda()
            sink = (torch.randn(H, generator=gen) * 3.0 + 3.0).float().cuda() if sinks else None
            meta = _meta(ops, [(s, n - m, m) for s, (n, m) in zip(slots, seqs)])
            got = ops.attention(q, meta, dataclasses.replace(view, v=view.k), H, 1.5 * D ** -0.5, window, sinks=sink)
            results[dtype, what] = got.float().cpu()
        ops.check_errors()
    for what in runs:
        assert rel_err(results[torch.bfloat16, what], results[torch.float32, what].double()) <= 1.5e-2, what
