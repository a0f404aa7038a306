"""Zevopel stacks (chunked attention with normed heads, sinks and gates; dense and routed feed-forwards; blocks that read the fp32 residual
stream itself and norm their outputs) against the plain restatement of tests/stack_oracle.py: every mechanism alone, whole models through
the engine's step function in all the ways a sequence can be cut up and batched, and generation through the public entry points.  The CPU
cases run the fp32 restatements of the device ops, the GPU cases the kernels in fp32 and bf16."""
import json
import math

import numpy as np
import pytest
import torch

import onnxruntime_genai_b200 as og
from onnxruntime_genai_b200 import ops
from onnxruntime_genai_b200.models import arch as A
from onnxruntime_genai_b200.models import moe
from onnxruntime_genai_b200.models.decoder import LayerWeights, PagedKVCache
from stack_harness import (BLOCK, RUNTIMES, close, dtype_of, feed, greedy_generation, mixed_batches, one_thread, open_engine, open_model, paged,  # noqa: F401
                           random_tokens, rewind_and_beams, rows_of, tol_of, wide_rows)
from stack_models import chunked, output_normed_stack, weights, write
from stack_oracle import (clamped_expert, gelu_feed_forward, rms_norm, rotary_frequencies, rotate, routed_experts, same_chunk, sink_attention, stack_forward,
                          wavelength_scaled)


@pytest.fixture(params=RUNTIMES)
def runtime(request):
    return request.param


# ------------------------------------------------------------------------------------------------ models
MIXED = output_normed_stack([chunked(), chunked(heads=6, kv_heads=3, dim=16, vdim=24, chunk=7, dims=6, ff=40, experts=8, top=3, scale=0.6),
                             chunked(heads=5, kv_heads=5, dim=40, vdim=40, chunk=33, ff=0, scaled=False, scale=0.3),
                             chunked(heads=8, kv_heads=1, dim=8, vdim=8, dims=8, chunk=1, ff=64, experts=4, top=1, limit=1.5),
                             chunked(heads=2, kv_heads=2, dim=32, vdim=8, chunk=64, dims=32, ff=72, experts=3, top=3, limit=0.4)])
# sizes no vector path can take: odd widths and head sizes, an odd number of rotated pairs, factors that are 1
ODD = output_normed_stack([chunked(heads=3, kv_heads=3, dim=9, vdim=5, dims=6, chunk=11, ff=13, scale=0.4),
                           chunked(heads=3, kv_heads=1, dim=7, vdim=3, dims=2, chunk=5, ff=7, experts=5, top=2, scale=0.4)],
                          vocab=37, width=45, eps=2e-2, residual_mult=1.0, embed_scale=1.0)
# every class of the tensor-core and warp-MMA attention kernels, experts on the grouped GEMMs, heads too wide for either
WIDE = output_normed_stack([chunked(heads=4, kv_heads=2, dim=128, vdim=56, chunk=48, dims=96, scale=0.15, ff=128),
                            chunked(heads=8, kv_heads=1, dim=64, vdim=128, chunk=100, dims=64, scale=0.2, ff=104, experts=12, top=4),
                            chunked(heads=2, kv_heads=2, dim=192, vdim=128, chunk=50, dims=128, scale=0.1, ff=0),
                            chunked(heads=3, kv_heads=1, dim=256, vdim=256, chunk=300, dims=32, scale=0.1, ff=70),
                            chunked(heads=4, kv_heads=4, dim=128, vdim=128, chunk=130, dims=128, scale=0.15, ff=200, experts=6, top=2),
                            chunked(heads=2, kv_heads=1, dim=72, vdim=200, chunk=16, dims=48, scale=0.2, ff=64),
                            chunked(heads=2, kv_heads=1, dim=264, vdim=24, chunk=90, dims=64, scale=0.1, ff=64)], vocab=160, width=128)
STACKS = {"zev_mixed": MIXED, "zev_odd": ODD, "zev_wide": WIDE}


# ------------------------------------------------------------------------------------------------ configuration
def test_config_is_read_into_layer_specs():
    a = A.from_stack_config(MIXED)
    assert a.model_type == "zevopel" and a.num_layers == 5 and not a.layernorm and not a.parallel_block and not a.pre_norm and a.layer_scale
    assert a.residual_multiplier == 0.6 and a.embed_scale == 1.7 and a.norm_eps == 3e-5 and a.norm_offset == 1.0
    sp = a.layer_specs
    assert [s.chunk for s in sp] == [20, 7, 33, 1, 64] and sp[0].qk_norm and sp[0].sinks and sp[0].head_gate and sp[2].ff == 0
    assert sp[1].moe == A.MoeSpec(8, 3, act="clamped", alpha=1.702, limit=0.7, weights="all") and sp[0].moe is None
    assert sp[2].rotary.scaling is None and sp[0].rotary.scaling["low"] == 1.0 and not a.has_linear_layers
    assert (a.num_heads, a.num_kv_heads, a.head_dim) == (8, 5, 40)
    shapes = A.stack_weight_shapes(a)
    assert "l2.norm2" not in shapes and "l2.ls2" not in shapes and shapes["l1.mlp.e7.down"] == (72, 40) and shapes["l1.mlp.router"] == (8, 72)
    assert shapes["l0.mix.g"] == (4, 72) and shapes["l0.mix.o"] == (72, 64) and shapes["l0.mix.k.norm"] == (24,)


@pytest.mark.parametrize("broken", [lambda c: c["layers"][0].update(type="delta"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                                    lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26),
                                    lambda c: c["layers"][1]["mlp"]["router"].update(top=9)])
def test_unknown_configurations_are_refused(broken):
    c = json.loads(json.dumps(MIXED))
    broken(c)
    with pytest.raises(ValueError):
        A.from_stack_config(c)


def test_wrong_and_missing_tensors_are_refused(tmp_path):
    w = weights(ODD)
    w["l1.mlp.e4.up"] = w["l1.mlp.e4.up"][:, :-1]
    with pytest.raises(ValueError, match="l1.mlp.e4.up"):
        og.Model(og.Config(write(ODD, w, tmp_path / "a"), provider="cpu"))
    w = weights(ODD)
    del w["l0.mix.sink"]
    with pytest.raises(ValueError, match="l0.mix.sink"):
        og.Model(og.Config(write(ODD, w, tmp_path / "b"), provider="cpu"))


def test_builder_exports_a_model_directory(tmp_path):
    from onnxruntime_genai_b200.models.builder import main
    d = write(ODD, weights(ODD, 3), tmp_path / "in")
    main(["-m", d, "-o", str(tmp_path / "out"), "-p", "bf16", "-e", "cpu", "--extra_options", "max_batch_size=3"])
    m = og.Model(str(tmp_path / "out"))
    assert m.type == "zevopel" and m.device_type == "cpu" and m.config.engine["dynamic_batching"]["max_batch_size"] == 3
    toks = random_tokens(ODD, 9)
    close(feed(open_engine(m), m, toks, [9]), stack_forward(ODD, weights(ODD, 3), toks)[0], 2e-4)
    main(["-m", d, "-o", str(tmp_path / "syn"), "-p", "fp32", "-e", "cpu", "--extra_options", "synthetic_weights=1", "seed=5"])
    og.Model(str(tmp_path / "syn"))


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("scaling", [dict(factor=4.0, original=64, low=1.0, high=4.0), dict(factor=8.0, original=8192, low=1.0, high=4.0),
                                     dict(factor=2.0, original=500, low=2.0, high=2.0), dict(factor=32.0, original=20, low=0.5, high=9.0), None])
@pytest.mark.parametrize("dims,base", [(8, 5000.0), (64, 500000.0), (6, 10.0)])
def test_rotary_tables(scaling, dims, base):
    rot = dict(dims=dims, base=base, scaling=scaling)
    f, amp = rotary_frequencies(rot)
    assert amp == 1.0
    cos, sin = A.rotary_tables(A.RotarySpec(dims, base, scaling), 400)
    for p in (0, 1, 17, 399):
        for i, fi in enumerate(f):
            assert cos[p, i] == pytest.approx(math.cos(p * fi), abs=1e-6) and sin[p, i] == pytest.approx(math.sin(p * fi), abs=1e-6)


def test_wavelength_scaling_has_three_ranges():
    s = dict(factor=8.0, original=1000.0, low=1.0, high=4.0)
    f = 2 * math.pi / np.array([100.0, 249.0, 251.0, 500.0, 999.0, 1001.0, 5000.0])
    got = A.wavelength_frequencies(f, s["factor"], s["original"], s["low"], s["high"])
    assert got == pytest.approx([wavelength_scaled(x, s) for x in f])
    assert got[1] == f[1] and got[5] == pytest.approx(f[5] / 8) and f[3] / 8 < got[3] < f[3]
    cfg = A.ArchConfig(rope_scaling=dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_position_embeddings=64),
                       head_dim=32, rope_theta=1000.0)
    mine = A.rotary_tables(A.RotarySpec(32, 1000.0, dict(factor=8.0, original=64, low=1.0, high=4.0)), 50)
    assert all(np.array_equal(a, b) for a, b in zip(mine, A.rope_caches(cfg, 50)))


@pytest.mark.parametrize("H", [24, 45, 512])
def test_scaled_embedding_in_two_types(runtime, H):
    dev, dt = runtime[0], dtype_of(runtime)
    table = torch.randn(11, H, generator=torch.Generator().manual_seed(H)).to(dt)
    ids = torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    h, x = ops.embedding_stream(ids.to(dev), table.to(dev), 0.3, dt)
    want = table[ids.long()].float() * 0.3
    assert h.dtype == torch.float32 and torch.equal(h.cpu(), want) and x.dtype == dt and torch.equal(x.cpu(), want.to(dt))


@pytest.mark.parametrize("T,H", [(3, 24), (5, 45), (1, 512), (70, 1000), (9, 4096), (2, 9000)])
def test_normed_output_joins_the_stream(runtime, T, H):
    """The stream keeps 32 bits: what is added to large values is exact, and the next sub-layer's input is its rounding."""
    g = torch.Generator().manual_seed(H)
    dev, dt = runtime[0], dtype_of(runtime)
    h, y, w = torch.randn(T, H, generator=g) * 300, (torch.randn(T, H, generator=g) * 2 + 1).to(dt), torch.randn(H, generator=g)
    want = h.double() + rms_norm(y.double(), w.double(), 0.7)
    hd = h.to(dev)
    x = ops.add_normed(hd, y.to(dev), w.to(dev), 0.7, dt)
    assert x.dtype == dt and torch.allclose(hd.cpu().double(), want, atol=2e-4, rtol=0)
    assert torch.equal(x.cpu(), hd.cpu().to(dt))


@pytest.mark.parametrize("T,inter,width", [(3, 64, 40), (5, 128, 128), (70, 21, 45), (300, 192, 128)])
def test_gelu_gated_feed_forward(runtime, T, inter, width):
    g = torch.Generator().manual_seed(T)
    dt, dev = dtype_of(runtime), runtime[0]
    x = (3 * torch.randn(T, width, generator=g)).to(dt)
    w = {n: (torch.randn(s, generator=g) / width ** 0.5).to(dt) for n, s in (("gate", (inter, width)), ("up", (inter, width)))}
    wi, il = torch.cat([w["gate"], w["up"]]), runtime == ("cuda", "bfloat16") and inter % 64 == 0
    got = ops.gate_up_act(x.to(dev), (ops.interleave_gate_up(wi) if il else wi).to(dev), None, "gelu_tanh", interleaved=il)
    w["down"] = torch.eye(inter)
    close(got, gelu_feed_forward(x.double(), {k: v.double() for k, v in w.items()}, ""), tol_of(runtime))


PREPS = [(4, 2, 24, 16, 16), (3, 3, 9, 5, 6), (5, 1, 128, 72, 80), (5, 5, 40, 40, 0), (2, 1, 264, 24, 264), (16, 4, 64, 128, 32), (8, 8, 8, 8, 2)]


@pytest.mark.parametrize("shape", PREPS, ids=lambda s: "x".join(map(str, s)))
def test_head_norms_rotation_and_append(runtime, shape):
    H, G, d, dv, rd = shape
    dev, dt = runtime[0], dtype_of(runtime)
    g = torch.Generator().manual_seed(d)
    kr, vr = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
    lens = [(0, 5), (30, 1), (15, 3), (200, 1)]
    pg = paged(lens, 20)
    T = sum(n for _, n in lens)
    q, k, v = (torch.randn(T, n, c, generator=g).to(dt) for n, c in ((H, d), (G, d), (G, dv)))
    qw, kw = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    rot = dict(dims=rd, base=300.0, scaling=dict(factor=4.0, original=100, low=1.0, high=4.0)) if rd else None
    fill = lambda x, c: torch.nn.functional.pad(x, (0, c - x.shape[-1])).reshape(T, -1)
    proj = torch.cat([fill(q, kr), fill(k, kr), fill(v, vr), torch.randn(T, 3, generator=g).to(dt)], 1)
    wide = wide_rows(proj, dev)
    kc, vc = torch.full((20 * BLOCK, G, kr), 7.0, dtype=dt, device=dev), torch.full((20 * BLOCK, G, vr), 7.0, dtype=dt, device=dev)
    cos = sin = None
    if rd:
        cos, sin = (torch.from_numpy(t).to(dev) for t in A.rotary_tables(A.RotarySpec(rd, 300.0, rot["scaling"]), 256))
    slots = pg["slots"].clone()
    slots[-1] = -1                                   # a token that is not kept
    ops.qkv_prep(wide, H, G, d, kr, vr, qw.to(dev), kw.to(dev), 1e-3, pg["pos"].to(dev), cos, sin, slots.to(dev), kc, vc)

    def want(x, w):
        y = rms_norm(x.double(), w.double(), 1e-3)
        full = torch.zeros(256, *y.shape[1:], dtype=torch.float64)
        out = torch.empty_like(y)
        for t, p in enumerate(pg["pos"].tolist()):   # rotate() counts positions from the first row
            full.zero_()
            full[p] = y[t]
            out[t] = rotate(full, rot)[p]
        return out
    got = wide.cpu()
    close(got[:, :H * kr].reshape(T * H, kr)[:, :d], want(q, qw).reshape(T * H, d), tol_of(runtime) / 4)
    kept = slots >= 0
    at = slots[kept].long()
    close(kc.cpu()[at][:, :, :d].reshape(-1, d), want(k, kw)[kept].reshape(-1, d), tol_of(runtime) / 4)
    assert torch.equal(vc.cpu()[at][:, :, :dv], v[kept]) and (kc.cpu()[at][:, :, d:] == 0).all()
    rest = torch.ones(20 * BLOCK, dtype=torch.bool)
    rest[at] = False
    assert (kc.cpu()[rest] == 7).all() and (vc.cpu()[rest] == 7).all() and torch.equal(got[:, -3:], proj[:, -3:])


SHAPES = [(4, 2, 24, 16), (3, 3, 16, 8), (6, 2, 128, 72), (8, 1, 64, 128), (2, 2, 128, 128), (4, 2, 96, 96), (3, 1, 192, 128), (2, 1, 256, 256), (2, 2, 72, 200),
          (2, 1, 264, 24), (20, 1, 40, 40)]


def _attention_case(shape, lens, chunk, seed, dt, needles=()):
    """Prepared queries, keys and values of requests (past, new).  needles (request, key, query): the query's heads point along the key, whose
    score then stands out."""
    H, G, d, dv = shape
    g = torch.Generator().manual_seed(seed)
    sink = torch.randn(H, generator=g)
    q, k, v, gate, want = [], [], [], [], []
    for b, (p, n) in enumerate(lens):
        T = p + n
        qq, kk, vv, gg = (torch.randn(T, *s, generator=g) for s in ((H, d), (G, d), (G, dv), (H,)))
        for nb, key, query in needles:
            if nb == b:
                u = kk[key] / kk[key].norm(dim=-1, keepdim=True)
                qq[query] = 9 * d ** 0.5 / kk[key].norm(dim=-1).mean() * u.repeat_interleave(H // G, 0)
        qq, kk, vv, gg = (t.to(dt) for t in (qq, kk, vv, gg))
        o = sink_attention(qq.double(), kk.double(), vv.double(), same_chunk(T, chunk) if chunk else torch.ones(T, T).tril().bool(), d ** -0.5, sink.double())
        want.append((o * torch.sigmoid(gg.double())[:, :, None]).reshape(T, H * dv)[p:])
        q.append(qq), k.append(kk), v.append(vv), gate.append(gg)
    return dict(q=q, k=k, v=v, gate=gate, sink=sink, want=torch.cat(want), scale=d ** -0.5)


def _run_attention(case, shape, lens, chunk, runtime, splits=None, order=None):
    H, G, d, dv = shape
    dev, dt = runtime[0], dtype_of(runtime)
    blocks = sum((p + n + BLOCK - 1) // BLOCK for p, n in lens) + 2
    pg = paged(lens, blocks, seed=5)
    kc, vc = torch.zeros(blocks * BLOCK, G, d, dtype=dt, device=dev), torch.zeros(blocks * BLOCK, G, dv, dtype=dt, device=dev)
    for b, (p, n) in enumerate(lens):
        kc[rows_of(pg, b, p + n).to(dev)], vc[rows_of(pg, b, p + n).to(dev)] = case["k"][b].to(dev), case["v"][b].to(dev)
    new = lambda x: torch.cat([t[p:] for t, (p, _) in zip(x, lens)])
    proj = torch.cat([new(case["q"]).reshape(-1, H * d), new(case["gate"])], 1)
    wide = wide_rows(proj, dev)
    t = {n: x.to(dev) for n, x in pg.items()}
    out = torch.full((proj.shape[0], H * dv), 5.0, dtype=dt, device=dev)
    ops.paged_attention(wide, kc, vc, t["cu"], t["past"], t["table"], BLOCK, H, G, d, case["scale"], 0, case["sink"].to(dev), 0.0,
                        max_q_len=max(n for _, n in lens), max_kv_len=max(p + n for p, n in lens), splits=splits, out=out, order=order, vdim=dv, chunk=chunk,
                        gate=wide[:, H * d:])
    if dev == "cuda":
        ops.check_kernel_status()
    return out


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("chunk", [0, 1, 23, 64, 150])
def test_chunked_attention_over_pages(runtime, shape, chunk):
    """Decode rows, short portions, and long prompts (beside short ones) with every split of the keys."""
    rng = np.random.RandomState(chunk)
    for lens in ([(0, 1), (70, 1), (15, 1), (16, 1), (299, 1), (300, 1)], [(0, 5), (31, 2), (40, 33), (17, 1)], [(0, 150), (5, 1), (131, 140), (400, 2)]):
        case = _attention_case(shape, lens, chunk, 3, dtype_of(runtime))
        order = torch.from_numpy(rng.permutation(len(lens)).astype(np.int32)).to(runtime[0])
        for splits, o in ((None, None), ((1, 0), order), ((3, 0), order), ((5, 64), None)):
            close(_run_attention(case, shape, lens, chunk, runtime, splits, o), case["want"], tol_of(runtime))


@pytest.mark.parametrize("chunk", [16, 33, 64])
@pytest.mark.parametrize("form", ["decode", "portion", "long"])
def test_chunk_edges_with_keys_that_stand_out(runtime, chunk, form):
    """One key dominates its query's scores: it decides the result when it lies in the query's run, and must not count when it is the last
    token of the run before; the same for the sequence's first tokens and at page borders."""
    shape = (4, 2, 56, 24)
    for q in sorted({0, 1, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 2 * chunk, 79, 80, 160}):
        start = q // chunk * chunk
        for key in sorted({0, start - 1, start, q - 1, q, max(0, q // BLOCK * BLOCK - 1)}):
            if not 0 <= key <= q:
                continue
            n = {"decode": 1, "portion": 7, "long": q + 1}[form]
            lens = [(max(0, q + 1 - n), min(n, q + 1)), (3, 2)]
            case = _attention_case(shape, lens, chunk, 11 + q + key, dtype_of(runtime), needles=[(0, key, q)])
            close(_run_attention(case, shape, lens, chunk, runtime), case["want"], tol_of(runtime))


def test_a_sink_takes_its_share(runtime):
    """Sinks far above every score leave almost nothing of the values, sinks far below leave the plain softmax."""
    shape, lens = (4, 2, 32, 24), [(0, 1), (40, 1), (0, 140), (3, 2)]
    for s in (30.0, -30.0):
        case = _attention_case(shape, lens, 50, 2, dtype_of(runtime))
        case["sink"].fill_(s)
        out = []
        for b, (p, n) in enumerate(lens):
            o = sink_attention(case["q"][b].double(), case["k"][b].double(), case["v"][b].double(), same_chunk(p + n, 50), case["scale"], case["sink"].double())
            out.append((o * torch.sigmoid(case["gate"][b].double())[:, :, None]).reshape(p + n, -1)[p:])
        got = _run_attention(case, shape, lens, 50, runtime)
        close(got, torch.cat(out), tol_of(runtime))
        assert (float(got.abs().max()) < 1e-6) == (s > 0)


EXPERTS = [(8, 3, 40, 72), (5, 2, 7, 45), (12, 4, 104, 128), (3, 3, 64, 64), (4, 1, 130, 40), (64, 6, 32, 128)]


@pytest.mark.parametrize("E,top,ff,W", EXPERTS)
@pytest.mark.parametrize("T", [1, 2, 40, 300])
def test_routed_experts(runtime, E, top, ff, W, T):
    """Inputs large enough that gates and ups are clamped on both sides; weights are probabilities among all experts."""
    g = torch.Generator().manual_seed(E * T)
    dev, dt = runtime[0], dtype_of(runtime)
    cfg = output_normed_stack([chunked(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, ff=ff, experts=E, top=top, limit=0.8)], vocab=4, width=W)
    w = {k: v for k, v in weights(cfg, seed=T).items()}
    x = (1.5 * torch.randn(T, W, generator=g)).to(dt)
    from onnxruntime_genai_b200.models.stack_checkpoint import build_stack_decoder
    model = build_stack_decoder(A.from_stack_config(cfg), lambda n: w[n], dev, dt)
    lw = model.layers[0]
    assert lw.exp_blocked == (runtime == ("cuda", "bfloat16") and W % 8 == 0)
    y = moe.moe_forward(model, lw, x.to(dev), defer=True)
    wd = {k: v.double() for k, v in w.items()}
    mlp = routed_experts(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    g_, u_ = x.double() @ wd["l0.mlp.e0.gate"].T, x.double() @ wd["l0.mlp.e0.up"].T
    assert T < 40 or ((g_ > 0.8).any() and (u_ > 0.8).any() and (u_ < -0.8).any() and (g_ < -0.8).any())
    h0 = torch.randn(T, W, generator=g)
    h = h0.clone().to(dev)
    wt = torch.rand(W, generator=g) + 0.5
    ops.add_normed(h, y, wt.to(dev), 1e-4, dt)
    close(h, h0.double() + rms_norm(mlp, wt.double(), 1e-4), tol_of(runtime) / 2)
    if isinstance(y, ops.PendingCombine):
        idx = torch.argsort(torch.softmax(x.double() @ wd["l0.mlp.router"].T, -1), descending=True)[:, :top]
        assert torch.equal(y.plan.topk_idx.cpu().long().sort(-1).values, idx.sort(-1).values)
        share = torch.softmax(x.double() @ wd["l0.mlp.router"].T, -1).gather(-1, idx).sort(-1).values
        assert torch.allclose(y.plan.topk_w.cpu().double().sort(-1).values, share, rtol=2e-5, atol=1e-7)


def test_expert_clamps_are_one_and_two_sided():
    x = torch.tensor([[4.0], [-4.0]], dtype=torch.float64)
    w = {"gate": torch.ones(1, 1).double(), "up": torch.ones(1, 1).double(), "down": torch.ones(1, 1).double()}
    a = A.MoeSpec(1, 1, act="clamped", limit=2.0)
    gu = torch.cat([x, x], 1)
    got = moe.swiglu_interleaved(gu, a.alpha, a.limit)
    assert torch.allclose(got, clamped_expert(x, w, "", 2.0), atol=1e-6)
    sg = lambda z: 1 / (1 + math.exp(-z))
    assert got[0, 0] == pytest.approx(2 * sg(1.702 * 2) * 3) and got[1, 0] == pytest.approx(-4 * sg(-1.702 * 4) * -1)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", list(STACKS))
def test_logits_of_a_whole_prompt(tmp_path_factory, runtime, name):
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    for n in (1, 2, 47, 150):
        toks = random_tokens(cfg, n, n)
        close(feed(open_engine(m), m, toks, [n]), stack_forward(cfg, w, toks)[0], tol_of(runtime))


@pytest.mark.parametrize("name", list(STACKS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 2, 17, 1, 1, 40], [100, 1], [64, 63, 2, 1], [15, 1, 1, 1, 16, 33], [19, 1, 2, 5, 1]], ids=str)
def test_portions_and_single_tokens(tmp_path_factory, runtime, name, cuts):
    """The same logits whatever the cut: token by token, pairs, ends and starts of pages and runs, long portions then decoding."""
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    toks = random_tokens(cfg, 130, 7)
    close(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], tol_of(runtime))


@pytest.mark.parametrize("name", list(STACKS))
def test_mixed_batches_reuse_pages(tmp_path_factory, runtime, name):
    mixed_batches(*open_model(tmp_path_factory, name, runtime, STACKS[name]), runtime)


def test_a_request_does_not_see_the_batch_around_it(tmp_path_factory, runtime):
    m, cfg, _ = open_model(tmp_path_factory, "zev_wide", runtime, WIDE)
    a, b, c = (random_tokens(cfg, n, s) for n, s in ((90, 1), (75, 2), (3, 3)))
    alone = feed(open_engine(m), m, a, [80, 1])
    eng = open_engine(m)
    ra, rb, rc = (og.Request(og.GeneratorParams(m)) for _ in range(3))
    rows = [eng.run_given([(rb, b[:70], []), (ra, a[:80], list(range(80))), (rc, c, [0])])[1]]
    for j in range(10):
        rows.append(eng.run_given([(ra, a[80 + j:81 + j], [0])] + ([(rb, b[70 + j:71 + j], [0])] if j < 5 else []))[0])
    close(torch.cat(rows), alone.double(), tol_of(runtime) / 4)


def test_short_portions_beside_single_tokens_of_long_requests(tmp_path_factory, runtime):
    """Keys of both are split between CTAs (few heads, long runs): neither launch may touch the rows of the other."""
    cfg = output_normed_stack([chunked(heads=2, kv_heads=2, dim=64, vdim=128, chunk=400, dims=32, scale=0.2, ff=64),
                               chunked(heads=2, kv_heads=1, dim=64, vdim=64, chunk=1000, dims=64, scale=0.2, ff=64)], width=64)
    m, cfg, w = open_model(tmp_path_factory, "zev_split", runtime, cfg)
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
    """Hundreds of single-token steps: runs end and begin among decoded tokens, pages fill up."""
    m, cfg, w = open_model(tmp_path_factory, "zev_mixed", runtime, MIXED)
    toks = random_tokens(cfg, 260, 9)
    close(feed(open_engine(m), m, toks, [20, 1]), stack_forward(cfg, w, toks)[0], tol_of(runtime))


def test_positions_count_from_the_first_token_of_the_sequence(tmp_path_factory, runtime):
    """Runs are counted from the sequence's start and not from a portion's: one token more in front moves every edge."""
    m, cfg, w = open_model(tmp_path_factory, "zev_mixed", runtime, MIXED)
    toks = random_tokens(cfg, 61, 30)
    for lead in (0, 1, 19, 20):
        t = np.concatenate([random_tokens(cfg, lead, 31), toks])
        close(feed(open_engine(m), m, t, [lead + 1, 30, 1, 2]), stack_forward(cfg, w, t)[0], tol_of(runtime))


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_through_generator_and_engine(tmp_path_factory, runtime):
    greedy_generation(*open_model(tmp_path_factory, "zev_wide", runtime, WIDE), runtime)


def test_batched_generator_rewind_and_beams(tmp_path_factory, runtime):
    rewind_and_beams(*open_model(tmp_path_factory, "zev_mixed", runtime, MIXED), runtime)


def test_sampled_generation_is_reproducible(tmp_path_factory, runtime):
    m, cfg, _ = open_model(tmp_path_factory, "zev_mixed", runtime, MIXED)
    out = []
    for _ in range(2):
        p = og.GeneratorParams(m)
        p.set_search_options(max_length=30, do_sample=True, top_k=20, temperature=0.8, random_seed=7)
        gen = og.Generator(m, p)
        gen.append_tokens(random_tokens(cfg, 8, 1).astype(np.int32).reshape(1, -1))
        while not gen.is_done():
            gen.generate_next_token()
        out.append(np.asarray(gen.get_sequence(0)).tolist())
    assert out[0] == out[1] and len(set(out[0][8:])) > 3


# ------------------------------------------------------------------------------------------------ cache sizes, trace replay
def test_cache_rows_follow_the_layers():
    a = A.from_stack_config(MIXED)
    kv = PagedKVCache(a, 3, BLOCK, "cpu", torch.float32)
    assert kv.full.numel() == 0 and kv.latent is None and kv.conv is None
    assert [tuple(t.shape[1:]) for t in kv.spec_kv[1]] == [(3, 16), (3, 24)] and kv.layer(0)[0].shape == (3 * BLOCK, 2, 24)
    per_token = 2 * (24 + 16) + 3 * (16 + 24) + 5 * 80 + 1 * 16 + 2 * 40
    assert PagedKVCache.bytes_per_block(a, BLOCK, torch.float32) == per_token * 4 * BLOCK
    assert sum(t.numel() for pools in kv.spec_kv.values() for t in pools) == per_token * 3 * BLOCK
    kv.spec_kv[2][1][BLOCK:2 * BLOCK] = 4.0
    kv.copy_blocks(torch.tensor([1]), torch.tensor([2]))
    assert (kv.spec_kv[2][1][2 * BLOCK:] == 4).all() and (kv.spec_kv[2][1][:BLOCK] == 0).all()
    with pytest.raises(RuntimeError, match="quantization"):
        PagedKVCache(a, 3, BLOCK, "cpu", torch.float32, kv_bits=8)


def test_layers_of_one_model_may_route_differently():
    """LayerWeights.moe overrides the model's rule."""
    a = A.ArchConfig(num_experts=4, experts_per_token=2, moe_style="standard", moe_norm_topk=False)
    assert a.moe_spec == A.MoeSpec(4, 2, act="silu", limit=7.0, weights="all")

    class Model:
        arch = a
    lw = LayerWeights(ln1_w=None, qkv_w=None, o_w=None, ln2_w=None)
    assert moe.spec_of(Model, lw).top == 2
    lw.moe = A.MoeSpec(8, 3)
    assert moe.spec_of(Model, lw).top == 3


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
