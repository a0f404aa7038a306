"""Tevilix stacks (parallel blocks with a norm per sub-layer, layers that run several times; windowed attention with mixed heads beside a gated average,
matrix memories; plain GELU feed-forwards and experts chosen in groups) against the plain restatement of tests/stack_oracle.py: every mechanism
alone, whole models through the engine's step function in all the ways a sequence can be cut up and batched, and generation through the public
entry points.  The CPU cases run the fp32 restatements of the device ops, the GPU cases the kernels in fp32 and bf16."""
import json
import math

import numpy as np
import pytest
import torch

import onnxruntime_genai_b200 as og
from onnxruntime_genai_b200 import ops
from onnxruntime_genai_b200.models import arch as A
from onnxruntime_genai_b200.models import moe
from onnxruntime_genai_b200.models.decoder import PagedKVCache
from onnxruntime_genai_b200.models.stack_checkpoint import build_stack_decoder
from stack_harness import (BLOCK, RUNTIMES, close, dtype_of, feed, greedy_generation, mixed_batches, one_thread, open_engine, open_model, paged,  # noqa: F401
                           random_tokens, rewind_and_beams, rows_of, tol_of, wide_rows)
from stack_models import grouped, memories, plain, side_by_side, two_norm_stack, weights, write
from stack_oracle import (gated_average, grouped_choice, grouped_experts, layer_norm, matrix_memory, mixed_heads_attention, mixed_scores, rms_norm,
                          rotate, stack_forward, visible)


@pytest.fixture(params=RUNTIMES)
def runtime(request):
    return request.param


def close_rows(got, want, runtime):
    """`close` for whole models.  With 16-bit projections a few rows may be further off: where a query nearly cancels against a memory, the norm of the head
    that follows makes up for the small result, and for its rounding."""
    if runtime[1] == "float32":
        return close(got, want, tol_of(runtime))
    err = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.std()
    assert torch.isfinite(err).all() and float(err.max()) < 4 * tol_of(runtime) and float((err > tol_of(runtime)).float().mean()) <= 0.02


# ------------------------------------------------------------------------------------------------ models
MIXED = two_norm_stack([memories(), side_by_side(mlp=grouped()), side_by_side(heads=6, kv_heads=3, dim=16, vdim=24, window=7, dims=16, factor=None, width=56,
                        scales=(1.3, 0.2)), memories(heads=2, dim=40, vdim=16, gate_cap=3.0, mlp=grouped(24, 8, 3, 4, 2, 0.7)), memories(mlp=None)], loop=(1, 3, 2))
# sizes no vector path can take: odd widths and head sizes, one key head, one rotated pair, groups of one expert
ODD = two_norm_stack([side_by_side(heads=3, kv_heads=1, dim=7, vdim=5, window=5, dims=2, width=13, mlp=plain(9)), memories(heads=3, dim=5, vdim=7, mlp=grouped(7, 3, 2, 3, 2)),
                      side_by_side(heads=3, kv_heads=3, dim=9, vdim=3, window=1, dims=0, width=1, mlp=None), memories(heads=1, dim=1, vdim=1, mlp=grouped(5, 1, 1, 1, 1))],
                     vocab=37, width=45, eps=2e-2, loop=(0, 2, 3), embed_scale=1.0)
# the classes of the tensor-core kernels: keys of all heads of 64 .. 512 columns and wider, memories of several widths; runs once
WIDE = two_norm_stack([side_by_side(heads=4, kv_heads=2, dim=128, vdim=128, window=70, dims=96, scale=0.12, width=256, mlp=grouped(128, 12, 4, 3, 2)),
                       memories(heads=2, dim=64, vdim=128, mlp=plain(256)),
                       side_by_side(heads=8, kv_heads=1, dim=64, vdim=56, window=33, dims=64, scale=0.15, width=130, mlp=None),
                       memories(heads=2, dim=128, vdim=64, mlp=grouped(72, 8, 2, 2, 1)),
                       side_by_side(heads=8, kv_heads=4, dim=128, vdim=64, window=100, dims=64, scale=0.1, width=64, mlp=plain(136)),
                       memories(heads=1, dim=24, vdim=264, mlp=None),
                       side_by_side(heads=4, kv_heads=4, dim=24, vdim=24, window=17, dims=24, scale=0.2, width=72, mlp=plain(64)),
                       side_by_side(heads=18, kv_heads=9, dim=64, vdim=16, window=40, dims=8, scale=0.15, width=24, mlp=None)],
                      vocab=160, width=128, loop=None)
STACKS = {"tev_mixed": MIXED, "tev_odd": ODD, "tev_wide": WIDE}


# ------------------------------------------------------------------------------------------------ configuration
def test_config_is_read_into_layer_specs():
    a = A.from_stack_config(MIXED)
    assert a.model_type == "tevilix" and a.layernorm and not a.norm_bias and a.parallel_block and a.sublayer_norms and not a.mlp_gated and a.embed_scale == 1.7
    sp = a.layer_specs
    assert a.num_layers == 7 and [s.source for s in sp] == [0, 1, 2, 1, 2, 3, 4] and [s.weights_of for s in sp] == [None, None, None, 1, 2, None, None]
    assert [s.kind for s in sp] == ["mlstm", "attention", "attention", "attention", "attention", "mlstm", "mlstm"] and a.has_linear_layers
    one = sp[1]
    assert one.talk and one.qk_norm and one.qkv_bias and one.o_bias and one.out_gate and one.window == 20 and one.prefix == "left." and one.mix_scale == 0.7
    assert one.rotary.scaling == {"factor": 5.0} and not one.rotary.neighbours and sp[2].rotary.scaling is None
    assert (one.beside.kind, one.beside.vdim, one.beside.mix_scale, one.beside.prefix) == ("min_gru", 40, 0.45, "right.")
    assert (sp[0].heads, sp[0].dim, sp[0].vdim, sp[0].gate_cap, sp[0].beside) == (3, 16, 24, 9.0, None)
    assert [s.state_elems for s in sp] == [3 * (16 * 24 + 17), 40, 56, 40, 56, 2 * (40 * 16 + 41), 3 * (16 * 24 + 17)] and a.recurrent_state_shape == (1364,)
    assert sp[5].moe == A.MoeSpec(8, 3, act="relu2", weights="sigmoid", groups=4, keep=2, scale=0.7) and not sp[5].moe.gated and sp[6].ff == 0
    shapes = A.stack_weight_shapes(a)
    assert shapes["l1.mix.left.talk"] == (4, 4) and shapes["l1.mix.left.o.b"] == (72,) and shapes["l1.mix.right.z.b"] == (40,) and shapes["l0.mix.i"] == (3, 72)
    assert shapes["l1.mlp.correction"] == (6,) and "l1.mlp.e0.gate" not in shapes and "l0.mlp.gate" not in shapes and "l0.norm1.b" not in shapes
    assert "l4.norm2" not in shapes and "l3.norm2" in shapes and "loop.step" not in shapes and "l5.norm1" not in shapes


@pytest.mark.parametrize("broken", [lambda c: c["layers"][0].update(type="delta"), lambda c: c["layers"][0]["mlp"].update(kind="gated"),
                                    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26),
                                    lambda c: c["layers"][1]["mlp"]["router"].update(top=4), lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4),
                                    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3), lambda c: c["loop"].update(stop=6),
                                    lambda c: c["loop"].update(times=0)])
def test_unknown_configurations_are_refused(broken):
    c = json.loads(json.dumps(MIXED))
    broken(c)
    with pytest.raises(ValueError):
        A.from_stack_config(c)


def test_wrong_and_missing_tensors_are_refused(tmp_path):
    for name, change in (("l0.mix.left.talk", None), ("l0.mix.right.x.b", lambda t: t[1:]), ("l1.mlp.correction", None), ("l1.mix.f.b", None), ("l2.mix.left.o.b", None),
                         ("l1.mlp.e2.up", lambda t: t[:1]), ("l0.norm2", None)):
        w = weights(ODD)
        if change:
            w[name] = change(w[name])
        else:
            del w[name]
        with pytest.raises(ValueError, match=name):
            og.Model(og.Config(write(ODD, w, tmp_path / name), provider="cpu"))


def test_builder_exports_a_model_directory(tmp_path):
    from onnxruntime_genai_b200.models.builder import main
    d = write(ODD, weights(ODD, 3), tmp_path / "in")
    main(["-m", d, "-o", str(tmp_path / "out"), "-p", "bf16", "-e", "cpu", "--extra_options", "max_batch_size=3"])
    m = og.Model(str(tmp_path / "out"))
    assert m.type == "tevilix" and m.device_type == "cpu" and m.config.engine["dynamic_batching"]["max_batch_size"] == 3
    toks = random_tokens(ODD, 9)
    close(feed(open_engine(m), m, toks, [9]), stack_forward(ODD, weights(ODD, 3), toks)[0], 2e-4)
    main(["-m", d, "-o", str(tmp_path / "syn"), "-p", "fp32", "-e", "cpu", "--extra_options", "synthetic_weights=1", "seed=5"])
    og.Model(str(tmp_path / "syn"))


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("T,H", [(3, 24), (5, 45), (1, 512), (70, 1000), (9, 4096)])
def test_sums_into_the_stream_and_two_norms(runtime, T, H):
    """One kernel adds rows (or the weighted experts' rows) to a stream that is far from zero mean and writes both sub-layers' norms."""
    g = torch.Generator().manual_seed(H)
    dev, dt = runtime[0], dtype_of(runtime)
    h, y, w1, w2 = 5 + torch.randn(T, H, generator=g) * 0.5, torch.randn(T, H, generator=g).to(dt), torch.randn(H, generator=g), torch.randn(H, generator=g)
    tol = 8e-3 if dt == torch.bfloat16 else 1e-5
    for add in (None, y):
        n = h.double() + (0 if add is None else add.double())
        hd = h.clone().to(dev)
        a, b = ops.norm_stream(hd, w1.to(dev), 1e-5, None, True, dt, add=None if add is None else add.to(dev), weight2=w2.to(dev))
        assert torch.allclose(hd.cpu().double(), n, atol=1e-5) and a.dtype == b.dtype == dt
        close(a, layer_norm(n, w1.double(), 0, 1e-5), tol)
        close(b, layer_norm(n, w2.double(), 0, 1e-5), tol)
        rows = torch.tensor([T - 1, 0], dtype=torch.int32)
        c = ops.norm_stream(h.clone().to(dev), w1.to(dev), 1e-5, None, True, dt, rows=rows.to(dev), add=None if add is None else add.to(dev))
        assert torch.equal(c.cpu(), a.cpu()[[T - 1, 0]])
    if dev == "cuda":
        plan = ops.moe_route(torch.randn(T, 5, generator=g).to(dev), 2, 1)
        ye = torch.randn(2 * T, H, generator=g).to(dt)
        hd = h.clone().to(dev)
        a, _ = ops.norm_stream(hd, w1.to(dev), 1e-5, None, True, dt, add=ops.PendingCombine(ye.to(dev), plan), weight2=w2.to(dev))
        n = h.double() + (ye.double()[plan.inv_pos.cpu().long()] * plan.topk_w.cpu().double()[:, :, None]).sum(1)
        assert torch.allclose(hd.cpu().double(), n, atol=1e-5)
        close(a, layer_norm(n, w1.double(), 0, 1e-5), tol)


@pytest.mark.parametrize("T,K,N", [(1, 72, 80), (5, 64, 256), (40, 128, 136), (300, 256, 1000), (3, 45, 9), (600, 128, 8192)])
@pytest.mark.parametrize("act", ["gelu_erf", "relu2", "silu", "gelu_tanh", "relu"])
def test_products_with_an_activation(runtime, T, K, N, act):
    g = torch.Generator().manual_seed(T)
    dev, dt = runtime[0], dtype_of(runtime)
    x, w = torch.randn(T, K, generator=g).to(dt), (1.5 * torch.randn(N, K, generator=g) / K ** 0.5).to(dt)
    y = x.double() @ w.double().T
    want = {"gelu_erf": 0.5 * y * (1 + torch.erf(y / math.sqrt(2))), "relu2": torch.relu(y) ** 2, "silu": y * torch.sigmoid(y), "relu": torch.relu(y),
            "gelu_tanh": 0.5 * y * (1 + torch.tanh(math.sqrt(2 / math.pi) * (y + 0.044715 * y ** 3)))}[act]
    out = torch.zeros(T, N + 11, dtype=dt, device=dev)
    ops.linear_act(wide_rows(x, dev), w.to(dev), act, out=out[:, 8:8 + N])
    close(out[:, 8:8 + N], want, 8e-3 if dt == torch.bfloat16 else 1e-5)
    assert (out[:, :8] == 0).all() and (out[:, -3:] == 0).all()


MIXES = [(4, 2, 24, 16, 16), (3, 1, 9, 5, 6), (5, 5, 128, 72, 80), (8, 2, 64, 128, 64), (6, 3, 40, 40, 0), (1, 1, 32, 8, 32), (32, 8, 128, 16, 32)]


@pytest.mark.parametrize("shape", MIXES, ids=lambda s: "x".join(map(str, s)))
def test_mixed_queries_have_the_scores_of_mixed_heads(runtime, shape):
    """Normed and rotated queries, mixed once per key head, against the mix of all heads' scores; keys and values go to the cache."""
    H, G, d, dv, rd = shape
    dev, dt = runtime[0], dtype_of(runtime)
    g = torch.Generator().manual_seed(d)
    kr, vr = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
    lens = [(0, 5), (30, 1), (15, 3), (200, 1)]
    pg = paged(lens, 20)
    T = sum(n for _, n in lens)
    q, k, v = (torch.randn(T, n, c, generator=g).to(dt) for n, c in ((H, d), (G, d), (G, dv)))
    qw, kw, talk = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g), torch.randn(H, H, generator=g)
    fill = lambda x, c: torch.nn.functional.pad(x, (0, c - x.shape[-1])).reshape(T, -1)
    wide = wide_rows(torch.cat([fill(q, kr), fill(k, kr), fill(v, vr), torch.randn(T, 3, generator=g).to(dt)], 1), dev)
    before = wide.clone()
    kc, vc = torch.full((20 * BLOCK, G, kr), 7.0, dtype=dt, device=dev), torch.full((20 * BLOCK, G, vr), 7.0, dtype=dt, device=dev)
    rot = dict(dims=rd, base=300.0, scaling=dict(factor=3.0)) if rd else None
    cos = sin = None
    if rd:
        cos, sin = (torch.from_numpy(t).to(dev) for t in A.rotary_tables(A.RotarySpec(rd, 300.0, rot["scaling"]), 256))
    slots = pg["slots"].clone()
    slots[-1] = -1
    mixed = torch.full((T, H * G * kr), 9.0, dtype=dt, device=dev)
    ops.qkv_prep(wide, H, G, d, kr, vr, qw.to(dev), kw.to(dev), 1e-5, pg["pos"].to(dev), cos, sin, slots.to(dev), kc, vc, talk=talk.to(dev), mixed=mixed)

    def turned(x, w):
        out = torch.empty(x.shape, dtype=torch.float64)
        for t, p in enumerate(pg["pos"].tolist()):         # rotate() counts positions from the first row
            full = torch.zeros(p + 1, *x.shape[1:], dtype=torch.float64)
            full[p] = rms_norm(x[t].double(), w.double(), 1e-5)
            out[t] = rotate(full, rot)[p]
        return out
    at = slots[slots >= 0].long()
    close(kc.cpu()[at][:, :, :d].reshape(-1, d), turned(k, kw)[slots >= 0].reshape(-1, d), tol_of(runtime) / 4)
    assert torch.equal(vc.cpu()[at][:, :, :dv], v[slots >= 0]) and (kc.cpu()[at][:, :, d:] == 0).all() and torch.equal(wide, before)
    rest = torch.ones(20 * BLOCK, dtype=torch.bool)
    rest[at] = False
    assert (kc.cpu()[rest] == 7).all() and (vc.cpu()[rest] == 7).all()
    keys = torch.randn(11, G, d, generator=g).double()
    got = torch.einsum("thcd,kcd->htk", mixed.cpu().double().view(T, H, G, kr)[..., :d], keys)
    want = mixed_scores(turned(q, qw), keys, talk.double(), 1.0)
    close(got.reshape(H, -1), want.reshape(H, -1), tol_of(runtime) / 4)
    assert (mixed.cpu().view(T, H, G, kr)[..., d:] == 0).all()


# (heads, key heads, key and value columns): keys of all heads together from one 16-byte piece to more than any tensor-core form takes
SHAPES = [(4, 2, 24, 16), (3, 3, 16, 8), (6, 2, 128, 72), (8, 1, 64, 128), (4, 2, 128, 128), (8, 4, 128, 128), (4, 4, 64, 64), (16, 4, 128, 64), (10, 5, 8, 40), (20, 1, 40, 40),
          (32, 4, 64, 64), (12, 3, 136, 24), (16, 8, 128, 32), (2, 2, 32, 264), (32, 8, 80, 64), (18, 6, 128, 136)]


def _attention_case(shape, lens, window, seed, dt, needles=(), loud=1.0):
    """Prepared queries, keys and values of requests (past, new).  needles (request, key, query): one score of one head stands out, and a mix brings it
    to all heads."""
    H, G, d, dv = shape
    g = torch.Generator().manual_seed(seed)
    q, k, v, gate, want = [], [], [], [], []
    talk = torch.eye(H) + 0.4 * torch.randn(H, H, generator=g)
    for b, (p, n) in enumerate(lens):
        T = p + n
        qq, kk, vv, gg = (torch.randn(T, *s, generator=g) for s in ((H, d), (G, d), (G, dv), (H * dv,)))
        qq = qq * loud
        for nb, key, query in needles:
            if nb == b:
                u = kk[key, 0] / kk[key, 0].norm()
                qq[query] = 0.3 * qq[query]
                qq[query, 0] = 14 * d ** 0.5 / kk[key, 0].norm() * u
                talk[:, 0] = 1.0
        # a query in the form in which it reaches the attention: mixed parts, one per key head
        parts = torch.einsum("hcg,tcgd->thcd", talk.view(H, G, H // G), qq.view(T, G, H // G, d)).reshape(T, H, G * d)
        parts, kk, vv, gg = (t.to(dt) for t in (parts, kk, vv, gg))
        q.append(parts), k.append(kk), v.append(vv), gate.append(gg)
        want.append((parts, qq))
    ok = [visible(p + n, dict(size=window) if window else None) for p, n in lens]
    outs = []
    for b, (p, n) in enumerate(lens):
        parts = want[b][0].double()
        s = torch.einsum("thx,kx->htk", parts, k[b].double().reshape(p + n, -1)) * d ** -0.5
        o = torch.einsum("htk,khv->thv", torch.softmax(s.masked_fill(~ok[b], -math.inf), -1), v[b].double().repeat_interleave(H // G, 1))
        outs.append(0.6 * (o.reshape(p + n, -1) * torch.sigmoid(gate[b].double()))[p:])
    return dict(q=q, raw=[x for _, x in want], talk=talk, k=k, v=v, gate=gate, want=torch.cat(outs), scale=d ** -0.5)


def _run_attention(case, shape, lens, window, runtime, splits=None, order=None):
    H, G, d, dv = shape
    dev, dt = runtime[0], dtype_of(runtime)
    blocks = sum((p + n + BLOCK - 1) // BLOCK for p, n in lens) + 2
    pg = paged(lens, blocks, seed=5)
    kc, vc = torch.zeros(blocks * BLOCK, G, d, dtype=dt, device=dev), torch.zeros(blocks * BLOCK, G, dv, dtype=dt, device=dev)
    for b, (p, n) in enumerate(lens):
        at = rows_of(pg, b, p + n).to(dev)
        kc[at], vc[at] = case["k"][b].to(dev), case["v"][b].to(dev)
    new = lambda x: torch.cat([t[p:] for t, (p, _) in zip(x, lens)])
    T = sum(n for _, n in lens)
    q = new(case["q"]).reshape(T, -1).to(dev).contiguous()
    gate = wide_rows(new(case["gate"]), dev)
    t = {n: x.to(dev) for n, x in pg.items()}
    out = torch.full((T, H * dv), 5.0, dtype=dt, device=dev)
    ops.paged_attention(q, kc, vc, t["cu"], t["past"], t["table"], BLOCK, H, G, G * d, case["scale"], window, max_q_len=max(n for _, n in lens),
                        max_kv_len=max(p + n for p, n in lens), splits=splits, out=out, order=order, vdim=dv, gate=gate, joint=True, out_scale=0.6)
    if dev == "cuda":
        ops.check_kernel_status()
    return out


def test_prepared_queries_are_the_mix_of_heads():
    """The form in which the cases below hold their queries against the plain mixed heads."""
    shape, lens = (6, 3, 8, 4), [(0, 30)]
    case = _attention_case(shape, lens, 9, 1, torch.float64)
    o = mixed_heads_attention(case["raw"][0].double(), case["k"][0], case["v"][0], visible(30, dict(size=9)), 8 ** -0.5, case["talk"].double())
    assert torch.allclose(0.6 * o.reshape(30, -1) * torch.sigmoid(case["gate"][0]), case["want"], atol=1e-6)


LENS = ([(0, 1), (70, 1), (15, 1), (16, 1), (299, 1), (300, 1)], [(0, 5), (31, 2), (40, 33), (17, 1)], [(0, 150), (5, 1), (131, 140), (400, 2)])


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [0, 1, 23, 64, 150])
def test_attention_with_mixed_heads_over_pages(runtime, shape, window):
    """Decode rows, short portions, and long prompts (beside short ones) with every split of the keys, a gate on every column."""
    rng = np.random.RandomState(window)
    for lens in LENS:
        case = _attention_case(shape, lens, window, 3, dtype_of(runtime), loud=2.0)
        order = torch.from_numpy(rng.permutation(len(lens)).astype(np.int32)).to(runtime[0])
        for splits, o in ((None, None), ((1, 0), order), ((3, 0), order), ((5, 64), None)):
            close(_run_attention(case, shape, lens, window, runtime, splits, o), case["want"], tol_of(runtime))


@pytest.mark.parametrize("shape", [(4, 2, 56, 24), (16, 4, 128, 64)], ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [16, 33, 64])
@pytest.mark.parametrize("form", ["decode", "portion", "long"])
def test_window_edges_with_keys_that_stand_out(runtime, window, form, shape):
    """One key dominates its query's scores in one head, and through the mix in all: it decides the result when it is the oldest one the window shows,
    and must not count when it is one older; the same for the sequence's first tokens and at page borders."""
    for q in sorted({0, 1, window - 1, window, window + 1, 2 * window, 79, 80, 160}):
        for key in sorted({0, q - window - 1, q - window, q - window + 1, q - 1, q, max(0, q // BLOCK * BLOCK - 1)}):
            if not 0 <= key <= q:
                continue
            n = {"decode": 1, "portion": 7, "long": q + 1}[form]
            lens = [(max(0, q + 1 - n), min(n, q + 1)), (3, 2)]
            case = _attention_case(shape, lens, window, 11 + q + key, dtype_of(runtime), needles=[(0, key, q)])
            close(_run_attention(case, shape, lens, window, runtime), case["want"], tol_of(runtime))


def _recurrent_steps(lens_of_steps, requests, slots):
    """Per step: cu_seqlens, past lengths, slots and the rows of every request."""
    done = [0] * requests
    for cuts in lens_of_steps:
        live = [(b, n) for b, n in enumerate(cuts) if n]
        t = lambda x: torch.tensor(np.asarray(x), dtype=torch.int32)
        yield live, t(np.cumsum([0] + [n for _, n in live])), t([done[b] for b, _ in live]), t([slots[b] for b, _ in live]), [done[b] for b, _ in live]
        for b, n in live:
            done[b] += n


STEPS = [[(70, 3, 1, 64), (1, 1, 1, 1), (5, 80, 2, 1), (17, 2, 66, 9), (1, 0, 1, 100), (2, 30, 1, 1)], [(1, 1, 1, 1)] * 6, [(600, 33, 0, 2), (1, 40, 129, 0), (3, 1, 1, 700)]]


@pytest.mark.parametrize("W", [1, 13, 24, 130, 384])
@pytest.mark.parametrize("steps", STEPS, ids=["portions", "single", "long"])
def test_gated_average(runtime, W, steps):
    """Portions of all sizes beside single tokens, states carried in slots that held something else; candidates on both sides of zero, gates that
    keep a state for hundreds of tokens and gates that replace it."""
    g = torch.Generator().manual_seed(W)
    dev, dt = runtime[0], dtype_of(runtime)
    n = [sum(s[b] for s in steps) for b in range(4)]
    z, x, o = ([(c * torch.randn(k, W, generator=g) + d).to(dt) for k in n] for c, d in ((3.0, -2.0), (1.5, 0.0), (1.0, 0.0)))
    want = [gated_average(torch.sigmoid(a.double()), b.double()) * c.double() * torch.sigmoid(c.double()) * 0.8 if len(a) else None for a, b, c in zip(z, x, o)]
    pool = torch.full((7, W + 5), 9.0, device=dev)
    state = pool[:, 2:2 + W]
    for live, cu, past, slots, at in _recurrent_steps(steps, 4, (5, 0, 3, 6)):
        rows = lambda t: torch.cat([t[b][a:a + k] for (b, k), a in zip(live, at)])
        up = (W + 7) // 8 * 8
        proj = torch.zeros(int(cu[-1]), 3 * up, dtype=dt, device=dev)
        for i, t in enumerate((z, x, o)):
            proj[:, i * up:i * up + W] = rows(t).to(dev)
        out = torch.full((int(cu[-1]), W + 6), 4.0, dtype=dt, device=dev)
        ops.min_gru(proj[:, :W], proj[:, up:up + W], proj[:, 2 * up:2 * up + W], state, slots.to(dev), cu.to(dev), past.to(dev), out[:, 4:4 + W], 0.8,
                    max(k for _, k in live))
        assert torch.allclose(out[:, 4:4 + W].cpu().double(), rows(want), **(dict(rtol=5e-3, atol=1e-5) if dt == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)))
        assert (out[:, :4] == 4).all() and (out[:, -2:] == 4).all()
    assert (pool[[1, 2, 4]] == 9).all() and (pool[:, :2] == 9).all() and (pool[:, 2 + W:] == 9).all()


def test_gated_average_keeps_a_state_in_32_bits(runtime):
    """Gates of 1e-3: a state moves by less than a 16-bit rounding step at a time, over many tokens and in both forms of a step."""
    g = torch.Generator().manual_seed(2)
    dev, dt = runtime[0], dtype_of(runtime)
    T, W = 900, 48
    z, x, o = (torch.full((T, W), -7.0) + 0.1 * torch.randn(T, W, generator=g)).to(dt), (3 + torch.randn(T, W, generator=g)).to(dt), torch.ones(T, W).to(dt)
    want = gated_average(torch.sigmoid(z.double()), x.double())
    proj = torch.cat([z, x, o], 1).to(dev)
    t = lambda *v: torch.tensor(v, dtype=torch.int32, device=dev)
    for cut in (900, 700, 1):
        state, got, at = torch.zeros(1, W, device=dev), [], 0
        while at < T:
            n = min(cut if cut > 1 or at < 880 else 1, T - at) if cut != 1 else (880 if at == 0 else 1)
            out = torch.empty(n, W, dtype=dt, device=dev)
            p = proj[at:at + n]
            ops.min_gru(p[:, :W], p[:, W:2 * W], p[:, 2 * W:], state, t(0), t(0, n), t(at), out, 1.0, n)
            got.append(out.float().cpu())
            at += n
        close(state.cpu(), want[-1:], 2e-3)
        factor = float(o[0, 0]) / (1 + math.exp(-1.0))
        close(torch.cat(got), want * factor, 1e-2 if dt == torch.bfloat16 else 1e-4)


MEMORIES = [(3, 16, 24), (2, 5, 7), (1, 1, 1), (2, 128, 128), (4, 64, 64), (2, 40, 264), (1, 256, 136), (2, 8, 520), (3, 24, 512)]


def _memory_case(shape, n, dt, seed, f_shift=2.0, i_shift=0.0, spread=1.0):
    """Raw projections and the plain result of requests of n[b] tokens."""
    H, d, dv = shape
    g = torch.Generator().manual_seed(seed)
    cap, eps = 8.0, 1e-4
    bias, norm = torch.randn(2 * H, generator=g) * 0.3, 1 + 0.2 * torch.randn(H * dv, generator=g)
    proj, gates, want = [], [], []
    for T in n:
        p = torch.randn(T, 2 * H * d + 2 * H * dv, generator=g).to(dt)
        z = spread * torch.randn(T, 2 * H, generator=g)
        z[:, :H] += i_shift
        z[:, H:] += f_shift
        q, k = (p[:, i * H * d:(i + 1) * H * d].double().view(T, H, d) for i in (0, 1))
        v, o = (p[:, 2 * H * d + i * H * dv:][:, :H * dv].double().view(T, H, dv) for i in (0, 1))
        y = cap * torch.tanh((z.double() + bias.double()) / cap)
        i, f = y[:, :H], -torch.log1p(torch.exp(-y[:, H:]))
        r = rms_norm(matrix_memory(q * d ** -0.5, k, v, i, f), 1.0, eps) * norm.double().view(H, dv) * torch.sigmoid(o) if T else q.new_zeros(0, H, dv)
        proj.append(p), gates.append(z), want.append(r.reshape(T, -1))
    return dict(proj=proj, gates=gates, want=want, bias=bias, norm=norm, cap=cap, eps=eps)


def _run_memories(case, shape, steps, runtime, tol, requests=4):
    H, d, dv = shape
    dev, dt = runtime[0], dtype_of(runtime)
    elems = H * (d * dv + d + 1)
    pool = torch.full((7, (elems + 3) // 4 * 4), 9.0, device=dev)
    for live, cu, past, slots, at in _recurrent_steps(steps, requests, (5, 0, 3, 6)):
        rows = lambda t: torch.cat([t[b][a:a + k] for (b, k), a in zip(live, at)])
        T = int(cu[-1])
        out = torch.full((T, H * dv + 8), 4.0, dtype=dt, device=dev)
        ops.mlstm(wide_rows(rows(case["proj"]), dev), rows(case["gates"]).to(dev), case["bias"].to(dev), H, d, dv, case["cap"], case["norm"].to(dev), case["eps"],
                  pool[:, :elems], slots.to(dev), cu.to(dev), past.to(dev), out[:, 4:4 + H * dv], max(k for _, k in live), min(k for _, k in live))
        close(out[:, 4:4 + H * dv], rows(case["want"]), tol)
        assert (out[:, :4] == 4).all() and (out[:, -4:] == 4).all()
    assert (pool[[1, 2, 4]] == 9).all()
    if dev == "cuda":
        ops.check_kernel_status()


@pytest.mark.parametrize("shape", MEMORIES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("steps", STEPS, ids=["portions", "single", "long"])
def test_matrix_memories(runtime, shape, steps):
    """Portions of all sizes beside single tokens, states carried in slots that held something else."""
    if shape[2] > 200 and steps is STEPS[2] and runtime[0] == "cpu":
        pytest.skip("the wide memories run long prompts on the GPU")
    case = _memory_case(shape, [sum(s[b] for s in steps) for b in range(4)], dtype_of(runtime), 3)
    _run_memories(case, shape, steps, runtime, 2e-2 if runtime[1] == "bfloat16" else 2e-4)


@pytest.mark.parametrize("f_shift,i_shift,spread", [(6.0, 0.0, 1.0), (-6.0, 0.0, 1.0), (0.0, -30.0, 2.0), (3.0, 30.0, 4.0), (2.0, -6.0, 8.0)],
                         ids=["keeps", "forgets", "closed", "open", "jumps"])
def test_memories_with_extreme_gates(runtime, f_shift, i_shift, spread):
    """Gates at their caps: states that live for hundreds of tokens, states that are gone at once (the maximum falls far below zero and the floor of the
    denominator decides), inputs that are hardly or fully let in, maxima that jump."""
    shape, steps = (2, 16, 24), [(130, 64, 1, 23), (1, 65, 2, 128), (70, 1, 40, 1)]
    case = _memory_case(shape, [sum(s[b] for s in steps) for b in range(4)], dtype_of(runtime), 5, f_shift, i_shift, spread)
    _run_memories(case, shape, steps, runtime, 2e-2 if runtime[1] == "bfloat16" else 3e-4)


def test_one_far_key_shows_in_a_memory(runtime):
    """A memory that is written once, far back, and only decays: its token still decides the output hundreds of tokens later, in every form of a step."""
    H, d, dv, T = 2, 16, 16, 400
    case = _memory_case((H, d, dv), [T], dtype_of(runtime), 1)
    for at in (0, 63, 64, 200):
        z = torch.full((T, 2 * H), -40.0)
        z[:, H:] = 9.0
        z[at, :H] = 5.0
        case["gates"][0] = z
        raw = case["proj"][0]
        raw[:, :H * d] = (0.3 * torch.randn(T, H * d, generator=torch.Generator().manual_seed(at)) + raw[at, H * d:2 * H * d].float()).to(raw.dtype)      # (queries that ask for it)
        p = raw.double()
        q, k, v, o = p[:, :H * d].view(T, H, d), p[:, H * d:2 * H * d].view(T, H, d), p[:, 2 * H * d:2 * H * d + H * dv].view(T, H, dv), p[:, 2 * H * d + H * dv:].view(T, H, dv)
        y = case["cap"] * torch.tanh((z.double() + case["bias"].double()) / case["cap"])
        r = matrix_memory(q * d ** -0.5, k, v, y[:, :H], -torch.log1p(torch.exp(-y[:, H:])))
        assert float((r[300:] / r[300:].norm(dim=-1, keepdim=True) * (v[at] / v[at].norm(dim=-1, keepdim=True))).sum(-1).abs().min()) > 0.95
        case["want"][0] = (rms_norm(r, 1.0, case["eps"]) * case["norm"].double().view(H, dv) * torch.sigmoid(o)).reshape(T, -1)
        for steps in ([(400,)], [(100,), (1,), (150,), (2,), (147,)], [(380,)] + [(1,)] * 20):
            _run_memories(case, (H, d, dv), steps, runtime, 3e-2 if runtime[1] == "bfloat16" else 3e-4, requests=1)


ROUTES = [(6, 2, 2, 1), (8, 3, 4, 2), (64, 6, 8, 4), (12, 4, 3, 2), (5, 5, 1, 1), (3, 2, 3, 2), (256, 8, 8, 4), (1, 1, 1, 1), (40, 4, 20, 19)]


@pytest.mark.parametrize("E,top,groups,keep", ROUTES)
def test_experts_are_chosen_in_groups_by_corrected_scores(runtime, E, top, groups, keep):
    """Corrections move the choice and not the weights; choice scores of both signs; a group's best pair counts, not its best expert."""
    g = torch.Generator().manual_seed(E)
    dev = runtime[0]
    logits, corr = 2 * torch.randn(200, E, generator=g), torch.randn(E, generator=g) - 0.8
    sp = A.MoeSpec(E, top, act="relu2", weights="sigmoid", groups=groups, keep=keep, scale=1.7)
    if dev == "cuda":
        plan = ops.moe_route(logits.to(dev), top, 3, correction=corr.to(dev), groups=groups, keep=keep, scale=1.7)
        w, ids = plan.topk_w.cpu(), plan.topk_idx.cpu().long()
    else:
        w, ids = moe.corrected_choice(logits, corr, sp)
    s = torch.sigmoid(logits.double())
    for t in range(200):
        want = grouped_choice(s[t] + corr.double(), groups, keep, top)
        assert sorted(ids[t].tolist()) == sorted(want.tolist())
        share = s[t, ids[t]] / s[t, ids[t]].sum() * 1.7
        assert torch.allclose(w[t].double(), share, rtol=1e-5)
    if 1 < groups < E and keep < groups:
        free = torch.stack([torch.topk(s[t] + corr.double(), top).indices.sort().values for t in range(200)])
        assert not torch.equal(free, ids.sort(-1).values) or keep * 20 > groups * 18


EXPERTS = [(8, 3, 40, 72, 4, 2), (6, 2, 7, 45, 2, 1), (12, 4, 104, 128, 3, 2), (64, 6, 32, 128, 8, 4), (1, 1, 24, 64, 1, 1), (4, 2, 130, 40, 2, 1)]


@pytest.mark.parametrize("E,top,ff,W,groups,keep", EXPERTS)
@pytest.mark.parametrize("T", [1, 2, 40, 300])
def test_squared_relu_experts(runtime, E, top, ff, W, groups, keep, T):
    g = torch.Generator().manual_seed(E * T)
    dev, dt = runtime[0], dtype_of(runtime)
    cfg = two_norm_stack([memories(heads=1, dim=8, vdim=8, mlp=grouped(ff, E, top, groups, keep, 1.6))], vocab=4, width=W, loop=None)
    w = weights(cfg, seed=T)
    x = torch.randn(T, W, generator=g).to(dt)
    wd = {k: v.double() for k, v in w.items()}
    model = build_stack_decoder(A.from_stack_config(cfg), lambda n: w[n], dev, dt)
    y = moe.moe_forward(model, model.layers[0], x.to(dev), defer=True)
    h0 = torch.randn(T, W, generator=g)
    h = h0.clone().to(dev)
    ops.norm_stream(h, torch.ones(W, device=dev), 1e-5, None, True, dt, add=y)
    c = torch.sigmoid(x.double() @ wd["l0.mlp.router"].T) + wd["l0.mlp.correction"]
    near = torch.zeros(T, dtype=torch.bool)
    for t in range(T):                                     # (cases that rounding decides do not count)
        pairs = c[t].view(groups, -1).sort(-1, descending=True).values[:, :2].sum(-1).sort(descending=True).values
        first = grouped_choice(c[t], groups, keep, min(top + 1, E // groups * keep))
        v = c[t, first].sort(descending=True).values
        near[t] = (keep < groups and pairs[keep - 1] - pairs[keep] < 2e-3) or (len(v) > top and v[top - 1] - v[top] < 2e-3)
    want = grouped_experts(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    assert float(near.float().mean()) < 0.2 or T <= 2
    if not near.all():
        close((h.cpu().double() - h0.double())[~near], want[~near], tol_of(runtime))


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", list(STACKS))
def test_logits_of_a_whole_prompt(tmp_path_factory, runtime, name):
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    for n in (1, 2, 47, 150):
        toks = random_tokens(cfg, n, n)
        close_rows(feed(open_engine(m), m, toks, [n]), stack_forward(cfg, w, toks)[0], runtime)


@pytest.mark.parametrize("name", list(STACKS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 2, 17, 1, 1, 40], [100, 1], [64, 63, 2, 1], [15, 1, 1, 1, 16, 33], [23, 24, 25, 1]], ids=str)
def test_portions_and_single_tokens(tmp_path_factory, runtime, name, cuts):
    """The same logits whatever the cut: token by token, pairs, ends and starts of pages, windows and chunks, long portions then decoding."""
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    toks = random_tokens(cfg, 130, 7)
    close_rows(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], runtime)


@pytest.mark.parametrize("name", list(STACKS))
def test_mixed_batches_reuse_pages_and_slots(tmp_path_factory, runtime, name):
    mixed_batches(*open_model(tmp_path_factory, name, runtime, STACKS[name]), runtime)


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 3, 2), (1, 2, 4), (2, 3, 2), (0, 1, 3)], ids=str)
def test_groups_of_layers_that_run_several_times(tmp_path_factory, runtime, loop):
    """Every pass has a cache and states of its own; layers around the group run once."""
    cfg = two_norm_stack([side_by_side(dims=8, mlp=grouped(24, 4, 1)), memories(), side_by_side(window=9, mlp=None)], loop=loop)
    m, cfg, w = open_model(tmp_path_factory, f"tev_loop{loop}", runtime, cfg)
    toks = random_tokens(cfg, 60, 3)
    for cuts in ([60], [23, 1, 1, 5]):
        close_rows(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], runtime)


def test_a_request_does_not_see_the_batch_around_it(tmp_path_factory, runtime):
    m, cfg, _ = open_model(tmp_path_factory, "tev_wide", runtime, WIDE)
    a, b, c = (random_tokens(cfg, n, s) for n, s in ((90, 1), (75, 2), (3, 3)))
    alone = feed(open_engine(m), m, a, [80, 1])
    eng = open_engine(m)
    ra, rb, rc = (og.Request(og.GeneratorParams(m)) for _ in range(3))
    rows = [eng.run_given([(rb, b[:70], []), (ra, a[:80], list(range(80))), (rc, c, [0])])[1]]
    for j in range(10):
        rows.append(eng.run_given([(ra, a[80 + j:81 + j], [0])] + ([(rb, b[70 + j:71 + j], [0])] if j < 5 else []))[0])
    close(torch.cat(rows), alone.double(), tol_of(runtime) / 4)


def test_short_portions_beside_single_tokens_of_long_requests(tmp_path_factory, runtime):
    """Keys of both are split between CTAs (few heads, long windows): neither launch may touch the rows of the other."""
    cfg = two_norm_stack([side_by_side(heads=2, kv_heads=1, dim=64, vdim=128, window=300, dims=32, scale=0.2, width=32, mlp=None),
                          side_by_side(heads=4, kv_heads=4, dim=64, vdim=64, window=250, dims=64, scale=0.2, width=32, mlp=None),
                          side_by_side(heads=4, kv_heads=4, dim=96, vdim=64, window=0, dims=64, scale=0.2, width=32, mlp=None)], width=64, loop=None)
    m, cfg, w = open_model(tmp_path_factory, "tev_split", runtime, cfg)
    seqs = [random_tokens(cfg, n, 60 + n) for n in (330, 212, 301)]
    eng = open_engine(m, tokens=1024)
    reqs = [og.Request(og.GeneratorParams(m)) for _ in seqs]
    eng.run_given([(r, t[:-10], []) for r, t in zip(reqs, seqs)])
    got, at = [[], [], []], [len(t) - 10 for t in seqs]
    for cut in ((1, 2, 1), (2, 1, 3), (1, 1, 2), (3, 3, 1), (1, 2, 2)):
        out = eng.run_given([(r, t[a:a + n], list(range(n))) for r, t, a, n in zip(reqs, seqs, at, cut)])
        for i, (o, n) in enumerate(zip(out, cut)):
            got[i].append(o.float().cpu())
            at[i] += n
    for t, g, a in zip(seqs, got, at):
        close(torch.cat(g), stack_forward(cfg, w, t)[0][len(t) - 10:a], tol_of(runtime))


def test_long_decoding(tmp_path_factory, runtime):
    """Hundreds of single-token steps: windows leave the prompt and then decoded tokens behind, states are carried on, pages fill up."""
    m, cfg, w = open_model(tmp_path_factory, "tev_mixed", runtime, MIXED)
    toks = random_tokens(cfg, 260, 9)
    close_rows(feed(open_engine(m), m, toks, [20, 1]), stack_forward(cfg, w, toks)[0], runtime)


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_through_generator_and_engine(tmp_path_factory, runtime):
    greedy_generation(*open_model(tmp_path_factory, "tev_wide", runtime, WIDE), runtime)


def test_batched_generator_rewind_and_beams(tmp_path_factory, runtime):
    rewind_and_beams(*open_model(tmp_path_factory, "tev_mixed", runtime, MIXED), runtime)


# ------------------------------------------------------------------------------------------------ cache sizes, trace replay
def test_cache_and_state_follow_the_runs_of_the_layers():
    a = A.from_stack_config(MIXED)
    kv = PagedKVCache(a, 3, BLOCK, "cpu", torch.float32)
    assert kv.full.numel() == 0 and kv.conv is None and kv.latent is None and sorted(kv.spec_kv) == [1, 2, 3, 4]
    assert [tuple(t.shape[1:]) for t in kv.spec_kv[1]] == [(2, 24), (2, 16)] and kv.spec_kv[1][0] is not kv.spec_kv[3][0]
    kv.ensure_state_slots(2)
    assert kv.state.shape == (7, 2, 1364) and kv.state_rows(1, beside=True).shape == (2, 40) and kv.state_rows(5).shape == (2, 1362)
    assert kv.state_rows(1).shape == (2, 0)
    per_token = 2 * (2 * (24 + 16) + 3 * (16 + 24))
    assert PagedKVCache.bytes_per_block(a, BLOCK, torch.float32) == per_token * 4 * BLOCK
    only = A.from_stack_config(two_norm_stack([memories()], loop=None))      # (no layer keeps rows: a block is still something)
    assert PagedKVCache.bytes_per_block(only, BLOCK, torch.float32) > 0 and PagedKVCache(only, 3, BLOCK, "cpu", torch.float32).spec_kv == {}


def test_trace_replay_writes_the_wanted_rows(tmp_path):
    from onnxruntime_genai_b200 import trace_replay
    cfg, w = ODD, weights(ODD, 8)
    m = og.Model(og.Config(write(cfg, w, tmp_path / "m"), provider="cpu"))
    eng = open_engine(m, blocks=8, batch=4, tokens=128)
    a, b = random_tokens(cfg, 30, 1).tolist(), random_tokens(cfg, 12, 2).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b[:11], "want": []}, {"id": "x", "tokens": a[20:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[21:], "want": [8]}, {"id": "y", "tokens": b[11:], "want": [0]}], "end": ["x", "y"]}]
    said = []
    trace_replay.replay(m, eng, [json.dumps(s) + "\n" for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists() and eng.core.free_blocks == 8
    wa, wb = stack_forward(cfg, w, a)[0], stack_forward(cfg, w, b)[0]
    close(torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(2, -1), wa[[0, 19]], 2e-4)
    close(torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")).view(2, -1), torch.stack([wa[29], wb[11]]), 2e-4)
