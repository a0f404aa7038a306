"""Sugelix stacks (hashed bigram embedding, tanh norms, layers that run several times; soft-capped, differential and latent attention with output
gates; routed and shared experts) against the plain restatement of tests/stack_oracle.py: every mechanism alone, whole models through the
engine's step function in all the ways a sequence can be cut up and batched, and generation through the public entry points.  The CPU cases
run the fp32 restatements of the device ops, the GPU cases the kernels in fp32 and bf16."""
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
from stack_models import capped, compressed_latent, differential, experts, looped_stack, weights, write
from stack_oracle import (bigram_rows, bounded_norm, clamped_expert, difference_factor, difference_of_maps, rms_norm, rotary_frequencies, rotate,
                          rotate_neighbours, selected_experts, sink_attention, softmax_attention, stack_forward, visible)


@pytest.fixture(params=RUNTIMES)
def runtime(request):
    return request.param


# ------------------------------------------------------------------------------------------------ models
MIXED = looped_stack([capped(), differential(), capped(heads=6, kv_heads=3, dim=16, vdim=24, dims=16, softcap=2.5, mlp=None), compressed_latent(),
                      differential(heads=3, kv_heads=3, dim=24, vdim=8, window=7, diff=0.75, dims=24, factor=1.0, mlp=experts(24, 8, 3, 1.2, 64, 0.5))],
                     loop=(1, 4, 2))
# sizes no vector path can take: odd widths and head sizes, one bucket, one rotated pair, one expert
ODD = looped_stack([differential(heads=3, kv_heads=1, dim=7, vdim=5, window=5, dims=2, mlp=experts(7, 3, 1)), capped(heads=3, kv_heads=3, dim=9, vdim=3, dims=6,
                   mlp=experts(5, 1, 1, 0.6, 11)), compressed_latent(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=13, q_rank=9, window=9, mlp=experts(7, 4, 2, 0.5, 0))],
                   vocab=37, width=45, eps=2e-2, buckets=1, loop=(0, 3, 3), embed_scale=1.0)
# the classes of the tensor-core and warp-MMA attention kernels, experts on the grouped GEMMs, heads too wide for either; runs once
WIDE = looped_stack([capped(heads=4, kv_heads=2, dim=128, vdim=128, dims=96, scale=0.12, softcap=5.0, mlp=experts(128, 12, 4)),
                     differential(heads=4, kv_heads=2, dim=64, vdim=128, window=70, dims=64, scale=0.15, mlp=experts(104, 5, 2, 0.9, 104, 0.9)),
                     compressed_latent(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=96, window=100, scale=0.1, mlp=experts(64, 4, 2, 0.7, 136)),
                     capped(heads=8, kv_heads=1, dim=64, vdim=56, dims=64, scale=0.15, softcap=30.0, mlp=None),
                     differential(heads=2, kv_heads=2, dim=128, vdim=256, window=33, dims=32, scale=0.1, mlp=experts(72, 3, 3)),
                     differential(heads=2, kv_heads=1, dim=136, vdim=40, window=90, dims=64, scale=0.1, mlp=None),
                     compressed_latent(heads=16, dim=16, rot_dim=16, vdim=32, kv_rank=64, q_rank=40, window=16, scale=0.2, mlp=None)],
                    vocab=160, width=128, buckets=97, mul_prev=1000003, mul_cur=999983, loop=None)
STACKS = {"sug_mixed": MIXED, "sug_odd": ODD, "sug_wide": WIDE}


# ------------------------------------------------------------------------------------------------ configuration
def test_config_is_read_into_layer_specs():
    a = A.from_stack_config(MIXED)
    assert a.model_type == "sugelix" and a.tanh_norm and a.pre_norm and not a.parallel_block and a.embed_scale == 1.7 and a.norm_eps == 3e-5
    assert a.bigram == dict(buckets=53, mul_prev=31, mul_cur=7) and a.passes == 2
    sp = a.layer_specs
    assert a.num_layers == 8 and [s.source for s in sp] == [0, 1, 2, 3, 1, 2, 3, 4] and [s.weights_of for s in sp] == [None] * 4 + [1, 2, 3, None]
    assert [s.opens_pass for s in sp] == [None, 0, None, None, 1, None, None, None]
    assert (sp[0].softcap, sp[0].window, sp[0].maps) == (6.0, 0, 1) and sp[0].rotary.neighbours and sp[0].qkv_bias and sp[0].out_gate and not sp[0].sinks
    assert (sp[1].maps, sp[1].diff, sp[1].window, sp[1].key_row, sp[1].softcap) == (2, 0.4, 20, 32, 0.0) and sp[1].rotary.scaling == {"factor": 3.0}
    assert sp[3].q_rank == 56 and sp[3].sinks and sp[3].window == 25 and not sp[3].rotary.neighbours and sp[2].ff == 0
    assert sp[7].moe == A.MoeSpec(8, 3, act="clamped", alpha=1.702, limit=1.2, weights="selected", shared_ff=64, shared_limit=0.5)
    shapes = A.stack_weight_shapes(a)
    assert shapes["bigram"] == (54, 72) and shapes["loop.step"] == (2, 72) and shapes["l0.norm1.alpha"] == () and "l2.norm2" not in shapes
    assert shapes["l1.mix.q"] == (128, 72) and shapes["l1.mix.k.b"] == (64,) and shapes["l1.mix.lq2"] == (16,) and "l0.mix.lq1" not in shapes
    assert shapes["l3.mix.uq"] == (144, 56) and "l3.mix.q" not in shapes and shapes["l4.mlp.shared.down"] == (72, 64) and "l5.norm1" not in shapes
    assert a.context_length == 32768


@pytest.mark.parametrize("broken", [lambda c: c["layers"][0].update(type="delta"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                                    lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26),
                                    lambda c: c["loop"].update(stop=6), lambda c: c["loop"].update(start=4, stop=4), lambda c: c["loop"].update(times=0)])
def test_unknown_configurations_are_refused(broken):
    c = json.loads(json.dumps(MIXED))
    broken(c)
    with pytest.raises(ValueError):
        A.from_stack_config(c)


def test_wrong_and_missing_tensors_are_refused(tmp_path):
    for name, change in (("l1.mix.lk1", None), ("loop.step", lambda t: t[:1]), ("l0.mix.q.b", lambda t: t[1:]), ("l2.mlp.e1.up", None), ("final.norm.alpha", None)):
        w = weights(ODD)
        if name == "l1.mix.lk1":
            name = "l0.mix.lk1"
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
    assert m.type == "sugelix" and m.device_type == "cpu" and m.config.engine["dynamic_batching"]["max_batch_size"] == 3
    toks = random_tokens(ODD, 9)
    close(feed(open_engine(m), m, toks, [9]), stack_forward(ODD, weights(ODD, 3), toks)[0], 2e-4)
    main(["-m", d, "-o", str(tmp_path / "syn"), "-p", "fp32", "-e", "cpu", "--extra_options", "synthetic_weights=1", "seed=5"])
    og.Model(str(tmp_path / "syn"))


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("factor", [1.0, 8.0, 2.5])
def test_linearly_scaled_rotary_tables(factor):
    rot = dict(dims=12, base=700.0, scaling=dict(factor=factor))
    f, amp = rotary_frequencies(rot)
    assert amp == 1.0 and f[0] == 1 / factor
    cos, sin = A.rotary_tables(A.RotarySpec(12, 700.0, rot["scaling"]), 400)
    for p in (0, 1, 17, 399):
        for i, fi in enumerate(f):
            assert cos[p, i] == pytest.approx(math.cos(p * fi), abs=1e-6) and sin[p, i] == pytest.approx(math.sin(p * fi), abs=1e-6)


def test_neighbouring_pairs_turn_like_halves_after_the_permutation():
    """Queries and keys permuted alike have the scores of the interleaved rotation; entries past the rotated ones stay."""
    rot = dict(dims=6, base=50.0)
    q, k = torch.randn(2, 9, 2, 11, dtype=torch.float64, generator=torch.Generator().manual_seed(0)).unbind(0)
    order = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9, 10]
    a = torch.einsum("ihd,jhd->hij", rotate_neighbours(q, rot), rotate_neighbours(k, rot))
    b = torch.einsum("ihd,jhd->hij", rotate(q[:, :, order], rot), rotate(k[:, :, order], rot))
    assert torch.allclose(a, b) and not torch.allclose(a, torch.einsum("ihd,jhd->hij", rotate(q, rot), rotate(k, rot)))
    assert torch.equal(rotate_neighbours(q, rot)[:, :, 6:], q[:, :, 6:])


@pytest.mark.parametrize("H", [24, 45, 512])
@pytest.mark.parametrize("spec", [dict(buckets=53, mul_prev=31, mul_cur=7), dict(buckets=1, mul_prev=3, mul_cur=5),
                                  dict(buckets=1009, mul_prev=2000003, mul_cur=1999993)], ids=lambda s: str(s["buckets"]))
def test_embedding_of_hashed_pairs(runtime, H, spec):
    """The token before a portion comes out of the pages, at page borders too; a first token has a row of its own."""
    dev, dt = runtime[0], dtype_of(runtime)
    g = torch.Generator().manual_seed(H)
    vocab = 3001
    table, big = torch.randn(vocab, H, generator=g).to(dt), torch.randn(spec["buckets"] + 1, H, generator=g).to(dt)
    lens = [(0, 5), (31, 1), (16, 3), (15, 2), (0, 1), (200, 40), (1, 1)]
    pg = paged(lens, 30)
    seqs = [torch.randint(0, vocab, (p + n,), generator=g, dtype=torch.int32) for p, n in lens]
    pool = torch.full((30 * BLOCK,), 77, dtype=torch.int32)
    for b, (p, _) in enumerate(lens):
        pool[rows_of(pg, b, p)] = seqs[b][:p]
    ids = torch.cat([s[p:] for s, (p, _) in zip(seqs, lens)])
    slots = pg["slots"].clone()
    slots[-1] = -1
    pd = pool.to(dev)
    got = ops.embedding_bigram(ids.to(dev), table.to(dev), 1.3, big.to(dev), spec, pd, slots.to(dev), pg["pos"].to(dev), pg["cu"].to(dev), pg["past"].to(dev),
                               pg["table"].to(dev), BLOCK)
    want = torch.cat([(table[s.long()].double() * 1.3 + big[bigram_rows(s.tolist(), **spec)].double())[p:] for s, (p, _) in zip(seqs, lens)])
    assert got.dtype == torch.float32 and torch.allclose(got.cpu().double(), want, atol=1e-6, rtol=1e-6)
    pool[slots[slots >= 0].long()] = ids[slots >= 0]
    assert torch.equal(pd.cpu(), pool)


def _tanh_norm(H, g):
    w = {"n": torch.randn(H, generator=g), "n.b": torch.randn(H, generator=g), "n.alpha": torch.tensor(0.37)}
    return ops.TanhNorm(w["n"], w["n.b"], 0.37), {k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("T,H", [(3, 24), (5, 45), (1, 512), (70, 1000), (9, 4096), (2, 9000)])
def test_sum_into_the_stream_and_its_tanh_norm(runtime, T, H):
    """Small entries, saturated ones, and a stream that keeps 32 bits; what is null is not added."""
    g = torch.Generator().manual_seed(H)
    dev, dt = runtime[0], dtype_of(runtime)
    norm, w = _tanh_norm(H, g)
    norm = ops.TanhNorm(norm.weight.to(dev), norm.bias.to(dev), norm.alpha)
    h = torch.randn(T, H, generator=g) * torch.logspace(-6, 2, H)
    y, first, step = torch.randn(T, H, generator=g).to(dt), torch.randn(T, H, generator=g), torch.randn(H, generator=g)
    for use in ((), ("y",), ("y", "step"), ("first", "step"), ("y", "first", "step")):
        kw = dict(first=first.to(dev) if "first" in use else None, step=step.to(dev) if "step" in use else None)
        n = h.double() + sum((t.double() for k, t in (("y", y), ("first", first), ("step", step)) if k in use), torch.zeros(()))
        hd = h.clone().to(dev)
        out = torch.empty_like(hd) if "first" in use else hd
        x = ops.add_tanh_norm(hd, y.to(dev) if "y" in use else None, norm, dt, out=out, **kw)
        assert x.dtype == dt and torch.allclose(out.cpu().double(), n, atol=2e-5, rtol=1e-6)
        assert torch.allclose(x.cpu().double(), bounded_norm(n, w, "n"), atol=1e-6 if dt == torch.float32 else 0, rtol=5e-6 if dt == torch.float32 else 8e-3) or \
            float((x.cpu().double() - bounded_norm(n, w, "n")).abs().max()) < (1e-6 if dt == torch.float32 else 2e-2)
        rows = torch.tensor([T - 1, 0], dtype=torch.int32)
        x2 = ops.add_tanh_norm(h.to(dev), y.to(dev) if "y" in use else None, norm, dt, rows=rows.to(dev), **kw)
        assert torch.equal(x2.cpu(), x.cpu()[[T - 1, 0]])
    tiny = torch.full((1, H), 1e-5).to(dev)
    zero = ops.TanhNorm(torch.ones(H).to(dev), torch.zeros(H).to(dev), 2.0)
    assert torch.allclose(ops.add_tanh_norm(tiny, None, zero, torch.float32).cpu(), torch.full((1, H), 2e-5), rtol=1e-5)


@pytest.mark.parametrize("T,heads,K,N", [(1, 3, 48, 24), (5, 4, 128, 64), (70, 2, 512, 128), (200, 3, 13, 7), (33, 5, 24, 20)])
def test_per_head_products_with_a_gate(runtime, T, heads, K, N):
    g = torch.Generator().manual_seed(T)
    dev, dt = runtime[0], dtype_of(runtime)
    x, w, gate = torch.randn(T, heads * K, generator=g).to(dt), (torch.randn(heads * N, K, generator=g) / K ** 0.5).to(dt), (2 * torch.randn(T, heads * N, generator=g)).to(dt)
    want = torch.cat([x[:, h * K:(h + 1) * K].double() @ w[h * N:(h + 1) * N].double().T for h in range(heads)], 1) * torch.sigmoid(gate.double())
    out = torch.zeros(T, heads * N + 5, dtype=dt, device=dev)
    ops.head_project(wide_rows(x, dev), w.to(dev), heads, K, out=out[:, 3:3 + heads * N], gate=wide_rows(gate, dev))
    close(out[:, 3:3 + heads * N], want, 8e-3 if dt == torch.bfloat16 else 1e-5)
    assert (out[:, :3] == 0).all() and (out[:, -2:] == 0).all()


@pytest.mark.parametrize("shape", [(4, 2, 24, 16, 16), (3, 1, 9, 5, 6), (5, 1, 128, 72, 80), (8, 2, 64, 128, 64), (6, 3, 40, 40, 0), (4, 4, 32, 8, 32)],
                         ids=lambda s: "x".join(map(str, s)))
def test_rotation_and_append_without_norms(runtime, shape):
    """Two key vectors per value head; a token whose slot is negative is not kept."""
    H, G, d, dv, rd = shape
    dev, dt = runtime[0], dtype_of(runtime)
    g = torch.Generator().manual_seed(d)
    kr, vr = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
    lens = [(0, 5), (30, 1), (15, 3), (200, 1)]
    pg = paged(lens, 20)
    T = sum(n for _, n in lens)
    q, k, v = (torch.randn(T, n, c, generator=g).to(dt) for n, c in ((2 * H, d), (2 * G, d), (G, dv)))
    fill = lambda x, c: torch.nn.functional.pad(x, (0, c - x.shape[-1])).reshape(T, -1)
    proj = torch.cat([fill(q, kr), fill(k, kr), fill(v, vr), torch.randn(T, 3, generator=g).to(dt)], 1)
    wide = wide_rows(proj, dev)
    kc, vc = torch.full((20 * BLOCK, G, 2 * kr), 7.0, dtype=dt, device=dev), torch.full((20 * BLOCK, G, vr), 7.0, dtype=dt, device=dev)
    rot = dict(dims=rd, base=300.0, scaling=dict(factor=3.0)) if rd else None
    cos = sin = None
    if rd:
        cos, sin = (torch.from_numpy(t).to(dev) for t in A.rotary_tables(A.RotarySpec(rd, 300.0, rot["scaling"]), 256))
    slots = pg["slots"].clone()
    slots[-1] = -1
    ops.qkv_prep(wide, 2 * H, 2 * G, d, kr, vr, None, None, 0.0, pg["pos"].to(dev), cos, sin, slots.to(dev), kc, vc, Hv=G)

    def want(x):
        out = torch.empty(x.shape, dtype=torch.float64)
        for t, p in enumerate(pg["pos"].tolist()):         # rotate() counts positions from the first row
            full = torch.zeros(p + 1, *x.shape[1:], dtype=torch.float64)
            full[p] = x[t].double()
            out[t] = rotate(full, rot)[p]
        return out
    got = wide.cpu()
    close(got[:, :2 * H * kr].reshape(T * 2 * H, kr)[:, :d], want(q).reshape(-1, d), tol_of(runtime) / 4)
    at = slots[slots >= 0].long()
    close(kc.cpu()[at].view(-1, 2 * G, kr)[:, :, :d].reshape(-1, d), want(k)[slots >= 0].reshape(-1, d), tol_of(runtime) / 4)
    assert torch.equal(vc.cpu()[at][:, :, :dv], v[slots >= 0]) and (kc.cpu()[at].view(-1, 2 * G, kr)[:, :, d:] == 0).all()
    rest = torch.ones(20 * BLOCK, dtype=torch.bool)
    rest[at] = False
    assert (kc.cpu()[rest] == 7).all() and (vc.cpu()[rest] == 7).all() and torch.equal(got[:, -3:], proj[:, -3:])


SHAPES = [(4, 2, 24, 16), (3, 3, 16, 8), (6, 2, 128, 72), (8, 1, 64, 128), (2, 2, 128, 128), (4, 2, 96, 96), (4, 4, 64, 64), (2, 1, 256, 256), (2, 1, 264, 24),
          (20, 1, 40, 40)]


def _attention_case(shape, lens, window, cap, seed, dt, needles=(), maps=1, loud=1.0):
    """Prepared queries, keys and values of requests (past, new).  needles (request, key, query): the query's vectors point along the key, whose
    score then stands out.  loud: factor on the queries."""
    H, G, d, dv = shape
    g = torch.Generator().manual_seed(seed)
    q, k, v, gate, want = [], [], [], [], []
    lam, diff = 0.63, 0.3
    for b, (p, n) in enumerate(lens):
        T = p + n
        qq, kk, vv, gg = (torch.randn(T, *s, generator=g) for s in ((H, maps, d), (G, maps, d), (G, dv), (H * dv,)))
        qq = qq * loud
        for nb, key, query in needles:
            if nb == b:
                u = kk[key] / kk[key].norm(dim=-1, keepdim=True)
                qq[query] = 9 * d ** 0.5 / kk[key].norm(dim=-1).mean() * u.repeat_interleave(H // G, 0)
                if maps == 2:
                    qq[query, :, 1] *= 0.05               # (the maps must not agree, or their difference says little)
        qq, kk, vv, gg = (t.to(dt) for t in (qq, kk, vv, gg))
        ok = visible(T, dict(size=window) if window else None)
        a = [softmax_attention(qq[:, :, m].double(), kk[:, :, m].double(), vv.double(), ok, d ** -0.5, cap) for m in range(maps)]
        o = a[0] if maps == 1 else difference_of_maps(*a, lam, diff, 1e-4)
        want.append((o.reshape(T, -1) * torch.sigmoid(gg.double()))[p:])
        q.append(qq), k.append(kk), v.append(vv), gate.append(gg)
    return dict(q=q, k=k, v=v, gate=gate, want=torch.cat(want), scale=d ** -0.5, diff=(lam, 1 - diff, 1e-4, dv) if maps == 2 else None)


def _run_attention(case, shape, lens, window, cap, runtime, splits=None, order=None, maps=1):
    H, G, d, dv = shape
    dev, dt = runtime[0], dtype_of(runtime)
    blocks = sum((p + n + BLOCK - 1) // BLOCK for p, n in lens) + 2
    pg = paged(lens, blocks, seed=5)
    kc, vc = torch.zeros(blocks * BLOCK, G, maps * d, dtype=dt, device=dev), torch.zeros(blocks * BLOCK, G, dv, dtype=dt, device=dev)
    for b, (p, n) in enumerate(lens):
        at = rows_of(pg, b, p + n).to(dev)
        kc[at], vc[at] = case["k"][b].reshape(p + n, G, -1).to(dev), case["v"][b].to(dev)
    new = lambda x: torch.cat([t[p:] for t, (p, _) in zip(x, lens)])
    T = sum(n for _, n in lens)
    wide = wide_rows(new(case["q"]).reshape(T, -1), dev)
    gate = wide_rows(new(case["gate"]), dev)
    t = {n: x.to(dev) for n, x in pg.items()}
    out = torch.full((T, H * dv), 5.0, dtype=dt, device=dev)
    ops.paged_attention(wide, kc, vc, t["cu"], t["past"], t["table"], BLOCK, H * maps, G, maps * d, case["scale"], window, None, cap,
                        max_q_len=max(n for _, n in lens), max_kv_len=max(p + n for p, n in lens), splits=splits, out=out, order=order, vdim=dv,
                        gate=gate, maps=maps, diff=case["diff"])
    if dev == "cuda":
        ops.check_kernel_status()
    return out


LENS = ([(0, 1), (70, 1), (15, 1), (16, 1), (299, 1), (300, 1)], [(0, 5), (31, 2), (40, 33), (17, 1)], [(0, 150), (5, 1), (131, 140), (400, 2)])


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window,cap", [(0, 0.0), (0, 1.5), (1, 0.0), (23, 4.0), (64, 0.0), (150, 30.0)])
def test_windowed_and_capped_attention_over_pages(runtime, shape, window, cap):
    """Decode rows, short portions, and long prompts (beside short ones) with every split of the keys, a gate on every column."""
    rng = np.random.RandomState(window)
    for lens in LENS:
        case = _attention_case(shape, lens, window, cap, 3, dtype_of(runtime), loud=3.0)
        order = torch.from_numpy(rng.permutation(len(lens)).astype(np.int32)).to(runtime[0])
        for splits, o in ((None, None), ((1, 0), order), ((3, 0), order), ((5, 64), None)):
            close(_run_attention(case, shape, lens, window, cap, runtime, splits, o), case["want"], tol_of(runtime))


@pytest.mark.parametrize("shape", [(4, 2, 16, 24), (3, 3, 8, 40), (6, 2, 64, 128), (2, 1, 128, 256), (4, 4, 64, 64), (2, 2, 136, 40), (2, 1, 40, 300), (10, 1, 24, 16)],
                         ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window,cap", [(0, 0.0), (1, 0.0), (23, 0.0), (64, 5.0), (150, 0.0)])
def test_differential_attention_over_pages(runtime, shape, window, cap):
    rng = np.random.RandomState(window)
    for lens in LENS:
        case = _attention_case(shape, lens, window, cap, 3, dtype_of(runtime), maps=2, loud=2.0)
        order = torch.from_numpy(rng.permutation(len(lens)).astype(np.int32)).to(runtime[0])
        for splits, o in ((None, None), ((1, 0), order), ((3, 0), order), ((5, 64), None)):
            close(_run_attention(case, shape, lens, window, cap, runtime, splits, o, maps=2), case["want"], tol_of(runtime))


@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("window", [16, 33, 64])
@pytest.mark.parametrize("form", ["decode", "portion", "long"])
def test_window_edges_with_keys_that_stand_out(runtime, window, form, maps):
    """One key dominates its query's scores: it decides the result when it is the oldest one the window shows, and must not count when it is one
    older; the same for the sequence's first tokens and at page borders."""
    shape = (4, 2, 56, 24)
    for q in sorted({0, 1, window - 1, window, window + 1, 2 * window, 79, 80, 160}):
        for key in sorted({0, q - window - 1, q - window, q - window + 1, q - 1, q, max(0, q // BLOCK * BLOCK - 1)}):
            if not 0 <= key <= q:
                continue
            n = {"decode": 1, "portion": 7, "long": q + 1}[form]
            lens = [(max(0, q + 1 - n), min(n, q + 1)), (3, 2)]
            case = _attention_case(shape, lens, window, 0.0, 11 + q + key, dtype_of(runtime), needles=[(0, key, q)], maps=maps)
            close(_run_attention(case, shape, lens, window, 0.0, runtime, maps=maps), case["want"], tol_of(runtime))


def test_capped_scores_saturate(runtime):
    """Scores far beyond the cap on both sides, around it, and far below it, where the cap hardly changes them."""
    shape, lens = (4, 2, 64, 64), [(0, 1), (90, 1), (0, 140), (30, 4)]
    for cap, loud in ((0.5, 40.0), (2.0, 2.0), (30.0, 20.0), (1000.0, 3.0)):
        case = _attention_case(shape, lens, 0, cap, 9, dtype_of(runtime), loud=loud)
        close(_run_attention(case, shape, lens, 0, cap, runtime), case["want"], tol_of(runtime))
        free = _attention_case(shape, lens, 0, 0.0, 9, dtype_of(runtime), loud=loud)
        assert (float((free["want"] - case["want"]).abs().max()) < 1e-3) == (cap == 1000.0)


def test_a_difference_that_nearly_cancels_is_still_normed(runtime):
    """A first token's maps agree (one visible key): the difference is (1 - lambda) times its value, and the norm makes up for its size."""
    shape, lens = (4, 2, 16, 32), [(0, 1), (0, 3), (0, 70)]
    case = _attention_case(shape, lens, 40, 0.0, 4, dtype_of(runtime), maps=2)
    lam, post, eps, dv = case["diff"]
    got = _run_attention(case, shape, lens, 40, 0.0, runtime, maps=2)
    v = case["v"][0][0].double().repeat_interleave(2, 0)
    first = (rms_norm((1 - lam) * v, 1.0, eps) * post).reshape(-1) * torch.sigmoid(case["gate"][0][0].double())
    close(got[:1], first[None], tol_of(runtime))
    close(got, case["want"], tol_of(runtime))


def test_factor_of_the_second_map():
    cfg = looped_stack([differential(heads=2, kv_heads=1, dim=16, vdim=8, diff=0.2)])
    w = weights(cfg, 5)
    m = build_stack_decoder(A.from_stack_config(cfg), lambda n: w[n], "cpu", torch.float32)
    want = float(difference_factor({k: v.double() for k, v in w.items()}, "l0.mix.", 0.2))
    assert m.layers[0].diff_lambda == pytest.approx(want, rel=1e-6) and abs(want - 0.2) > 0.02 and m.layers[1] is m.layers[0]


LATENTS = [(3, 40, 8, 24, 48, 56), (4, 64, 32, 64, 128, 96), (16, 16, 16, 32, 64, 40), (3, 5, 6, 7, 13, 9), (2, 128, 64, 128, 256, 200), (5, 8, 2, 16, 24, 8)]


@pytest.mark.parametrize("shape", LATENTS, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [0, 1, 30, 100])
def test_compressed_latent_layer(runtime, shape, window):
    """The whole mixer in every form of a step (decode, short portions, long prompts beside them) over pages; sinks of both signs."""
    H, d, r, dv, R, Q = shape
    e = compressed_latent(H, d, r, dv, R, Q, window, scale=(d + r) ** -0.5, mlp=None)
    cfg = looped_stack([e, differential(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, mlp=None)], width=64, loop=None)
    w = weights(cfg, R)
    w["l0.mix.sink"] = (torch.arange(H) % 3 * 2.0 - 1.0).to(torch.bfloat16)
    w["l0.mix.uq"] = w["l0.mix.uq"] * 3
    a = A.from_stack_config(cfg)
    dev, dt = runtime[0], dtype_of(runtime)
    model = build_stack_decoder(a, lambda n: w[n], dev, dt)
    from onnxruntime_genai_b200.models.decoder import StepInputs
    wd = {k: v.double() for k, v in w.items()}
    from stack_oracle import compressed_latent_mixer
    g = torch.Generator().manual_seed(window)
    T = 190
    xs = [torch.randn(T, 64, generator=g).to(dt) for _ in range(4)]
    want = [compressed_latent_mixer(x.double(), wd, "l0.mix.", e["mixer"], cfg["norm"]["eps"]) for x in xs]
    kv = PagedKVCache(a, 60, BLOCK, dev, dt)
    done = [0] * 4
    for cuts in ((70, 3, 1, 64), (1, 1, 1, 1), (5, 80, 2, 1), (17, 2, 66, 9), (1, 30, 1, 100)):
        lens = list(zip(done, cuts))
        full = paged([(0, T)] * 4, 60, seed=3)
        pos = np.concatenate([np.arange(p, p + n) for p, n in lens])
        slots = np.concatenate([full["table"].numpy()[b][np.arange(p, p + n) // BLOCK] * BLOCK + np.arange(p, p + n) % BLOCK for b, (p, n) in enumerate(lens)])
        t = lambda v: torch.tensor(np.asarray(v), dtype=torch.int32, device=dev)
        s = StepInputs(input_ids=t(pos), positions=t(pos), slot_mapping=t(slots), cu_seqlens=t(np.cumsum([0] + list(cuts))), past_lens=t(done),
                       block_table=full["table"].to(dev), max_q_len=max(cuts), max_kv_len=max(p + n for p, n in lens), host_lens=lens)
        x = torch.cat([xs[b][p:p + n] for b, (p, n) in enumerate(lens)]).to(dev)
        out = torch.empty(x.shape[0], H * dv, dtype=dt, device=dev)
        model._latent_attention(s, kv, 0, model.layers[0], x, out)
        got = ops.linear(out, model.layers[0].o_w)
        close(got, torch.cat([want[b][p:p + n] for b, (p, n) in enumerate(lens)]), tol_of(runtime))
        done = [p + n for p, n in lens]
    if dev == "cuda":
        ops.check_kernel_status()


def test_latent_window_edges_and_sinks(runtime):
    """A latent whose key stands out just inside and just outside the window, beside a sink that leaves little or nothing of the values."""
    H, d, r, R, window = 4, 32, 16, 64, 24
    sh = ops.latent_shape(H, d, r, 32, R, 0)
    dev, dt = runtime[0], dtype_of(runtime)
    g = torch.Generator().manual_seed(1)
    for sink in (-20.0, 1.0, 40.0):
        sinks = torch.full((H,), sink)
        for q, key in ((60, 60 - window + 1), (60, 60 - window), (60, 48), (60, 47), (23, 0), (24, 0), (15, 0), (40, 39)):
            pg = paged([(q, 1), (0, 2)], 8)
            rows = torch.randn(q + 1, R + r, generator=g).to(dt)
            qv = torch.randn(3, H, R + r, generator=g)
            qv[0] = 40 * rows[key].float() / rows[key].float().norm() ** 2
            qv = qv.to(dt)
            cache = torch.zeros(8 * BLOCK, R + r, dtype=dt)
            cache[rows_of(pg, 0, q + 1)] = rows
            other = torch.randn(2, R + r, generator=g).to(dt)
            cache[rows_of(pg, 1, 2)] = other
            full = torch.zeros(3, H, d + r, dtype=dt)
            full[:, :, d:] = qv[:, :, R:]
            t = {n: x.to(dev) for n, x in pg.items()}
            for splits in (None, 3):
                got = ops.latent_attention(qv[:, :, :R].reshape(3, -1).contiguous().to(dev), wide_rows(full.reshape(3, -1), dev), sh, cache.to(dev), t["cu"], t["past"],
                                           t["table"], BLOCK, 1.0, window, 2, q + 1, splits=splits, sinks=sinks.to(dev))
                vis = rows[max(0, q - window + 1):].double()
                want = sink_attention(qv[:1].double(), vis[:, None].expand(-1, 1, -1), vis[:, None, :R], torch.ones(1, len(vis), dtype=torch.bool), 1.0, sinks.double())
                w2 = sink_attention(qv[1:].double(), other.double()[:, None], other.double()[:, None, :R], visible(2, None), 1.0, sinks.double())
                both = torch.cat([want, w2]).reshape(3, -1)
                assert float((got.cpu().double() - both).abs().max()) < 8 * tol_of(runtime) * max(0.01, float(both.abs().max()))


EXPERTS = [(8, 3, 40, 72, None, None), (5, 2, 7, 45, None, None), (12, 4, 104, 128, 104, 0.8), (3, 3, 64, 64, 72, None), (4, 1, 130, 40, 130, 0.3), (64, 6, 32, 128, 0, None),
           (1, 1, 24, 64, None, None), (5, 2, 7, 45, 9, 1.1)]


@pytest.mark.parametrize("E,top,ff,W,shared,limit", EXPERTS)
@pytest.mark.parametrize("T", [1, 2, 40, 300])
def test_selected_and_shared_experts(runtime, E, top, ff, W, shared, limit, T):
    """Inputs large enough that gates and ups are clamped on both sides; a shared expert stacked with the others or beside them."""
    g = torch.Generator().manual_seed(E * T)
    dev, dt = runtime[0], dtype_of(runtime)
    cfg = looped_stack([capped(heads=1, kv_heads=1, dim=8, vdim=8, dims=8, mlp=experts(ff, E, top, 0.8, shared, limit))], vocab=4, width=W, loop=None)
    w = weights(cfg, seed=T)
    x = (1.5 * torch.randn(T, W, generator=g)).to(dt)
    wd = {k: v.double() for k, v in w.items()}
    z = x.double() @ wd["l0.mlp.router"].T
    model = build_stack_decoder(A.from_stack_config(cfg), lambda n: w[n], dev, dt)
    lw = model.layers[0]
    assert lw.exp_shared == (shared != 0 and (shared or ff) == ff and (limit or 0.8) == 0.8) and (lw.shared_gate_up_w is not None) == (shared != 0 and not lw.exp_shared)
    y = moe.moe_forward(model, lw, x.to(dev), defer=True)
    norm, nw = _tanh_norm(W, g)
    norm = ops.TanhNorm(norm.weight.to(dev), norm.bias.to(dev), norm.alpha)
    h0 = torch.randn(T, W, generator=g)
    h = h0.clone().to(dev)
    ops.add_tanh_norm(h, y, norm, dt, out=h)
    want = selected_experts(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    near = (torch.topk(z, min(top + 1, E), -1).values.diff(dim=-1)[:, -1].abs() < 1e-4) if E > top else torch.zeros(T, dtype=torch.bool)
    close((h.cpu().double() - h0.double())[~near], want[~near], tol_of(runtime))
    if isinstance(y, ops.PendingCombine):
        share = torch.softmax(torch.topk(z, top, -1).values, -1).sort(-1).values
        assert torch.allclose(y.plan.topk_w.cpu().double()[:, :top].sort(-1).values[~near], share[~near], rtol=2e-5, atol=1e-6)
        if lw.exp_shared:
            assert (y.plan.topk_idx[:, top] == E).all() and (y.plan.topk_w[:, top] == 1).all()


def test_shared_expert_has_its_own_limit():
    cfg = looped_stack([capped(mlp=experts(16, 2, 1, 0.5, 16, 2.0))], width=32, loop=None)
    w = {k: v.double() for k, v in weights(cfg, 2).items()}
    x = 3 * torch.randn(5, 32, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    m = cfg["layers"][0]["mlp"]
    a = selected_experts(x, w, "l0.mlp.", m) - selected_experts(x, w, "l0.mlp.", dict(m, shared=None))
    assert torch.allclose(a, clamped_expert(x, w, "l0.mlp.shared.", 2.0)) and not torch.allclose(a, clamped_expert(x, w, "l0.mlp.shared.", 0.5))


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
    """The same logits whatever the cut: token by token, pairs, ends and starts of pages and windows, long portions then decoding."""
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    toks = random_tokens(cfg, 130, 7)
    close(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], tol_of(runtime))


@pytest.mark.parametrize("name", list(STACKS))
def test_mixed_batches_reuse_pages(tmp_path_factory, runtime, name):
    mixed_batches(*open_model(tmp_path_factory, name, runtime, STACKS[name]), runtime)


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 3, 2), (1, 2, 4), (2, 3, 2), (0, 1, 3)], ids=str)
def test_groups_of_layers_that_run_several_times(tmp_path_factory, runtime, loop):
    """Every pass has a cache of its own, a vector of its own, and (but the first) the embedding output; layers around the group run once."""
    cfg = looped_stack([capped(dims=8, mlp=experts(24, 3, 1)), differential(window=9), compressed_latent(window=11, mlp=None)], loop=loop)
    m, cfg, w = open_model(tmp_path_factory, f"sug_loop{loop}", runtime, cfg)
    toks = random_tokens(cfg, 60, 3)
    for cuts in ([60], [23, 1, 1, 5]):
        close(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], tol_of(runtime))
    if loop and loop[2] > 1 and runtime[1] == "float32":
        for drop in range(loop[2]):                         # (every pass's vector shows in the logits)
            w2 = dict(w)
            w2["loop.step"] = w["loop.step"].clone()
            w2["loop.step"][drop] = 0
            assert float((stack_forward(cfg, w2, toks)[0] - stack_forward(cfg, w, toks)[0]).std()) > 0.05 * float(stack_forward(cfg, w, toks)[0].std())


def test_a_request_does_not_see_the_batch_around_it(tmp_path_factory, runtime):
    m, cfg, _ = open_model(tmp_path_factory, "sug_wide", runtime, WIDE)
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
    cfg = looped_stack([differential(heads=1, kv_heads=1, dim=64, vdim=128, window=300, dims=32, scale=0.2, mlp=None),
                        capped(heads=2, kv_heads=1, dim=64, vdim=64, dims=64, scale=0.2, mlp=None),
                        compressed_latent(heads=2, window=250, mlp=None)], width=64, loop=None)
    m, cfg, w = open_model(tmp_path_factory, "sug_split", runtime, cfg)
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


def test_the_token_before_a_portion_is_kept_with_the_pages(tmp_path_factory, runtime):
    """Two requests with different tokens before the same ones, cut at page borders and inside pages, on pages used before: the pair decides."""
    cfg = looped_stack([capped(dims=8, mlp=None)], buckets=401, loop=None)
    w = weights(cfg, 6)
    w["bigram"] = w["bigram"] * 3
    m, cfg, w = open_model(tmp_path_factory, "sug_pairs", runtime, cfg, w)
    eng = open_engine(m, blocks=8, batch=3)
    for seed in range(3):
        for cut in (1, 15, 16, 17, 32):
            a, b = random_tokens(cfg, 48, seed), random_tokens(cfg, 48, 90 + seed)
            b[cut:] = a[cut:]
            ra, rb = og.Request(og.GeneratorParams(m)), og.Request(og.GeneratorParams(m))
            eng.run_given([(ra, a[:cut], []), (rb, b[:cut], [])])
            ga, gb = eng.run_given([(ra, a[cut:], [0, 5]), (rb, b[cut:], [0, 5])])
            close(ga, stack_forward(cfg, w, a)[0][[cut, cut + 5]], tol_of(runtime))
            close(gb, stack_forward(cfg, w, b)[0][[cut, cut + 5]], tol_of(runtime))
            eng.remove_request(ra), eng.remove_request(rb)


def test_long_decoding(tmp_path_factory, runtime):
    """Hundreds of single-token steps: windows leave the prompt and then decoded tokens behind, pages fill up."""
    m, cfg, w = open_model(tmp_path_factory, "sug_mixed", runtime, MIXED)
    toks = random_tokens(cfg, 260, 9)
    close(feed(open_engine(m), m, toks, [20, 1]), stack_forward(cfg, w, toks)[0], tol_of(runtime))


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_through_generator_and_engine(tmp_path_factory, runtime):
    greedy_generation(*open_model(tmp_path_factory, "sug_wide", runtime, WIDE), runtime)


def test_batched_generator_rewind_and_beams(tmp_path_factory, runtime):
    rewind_and_beams(*open_model(tmp_path_factory, "sug_mixed", runtime, MIXED), runtime)


def test_token_ids_cannot_be_replaced_by_embeddings():
    m = build_stack_decoder(A.from_stack_config(ODD), lambda n, w=weights(ODD): w[n], "cpu", torch.float32)
    from onnxruntime_genai_b200.models.decoder import StepInputs
    z = torch.zeros(1, dtype=torch.int32)
    s = StepInputs(z, z, z, torch.tensor([0, 1], dtype=torch.int32), z, torch.zeros(1, 1, dtype=torch.int32), inputs_embeds=torch.zeros(1, 45))
    with pytest.raises(RuntimeError, match="token ids"):
        m.forward(s, PagedKVCache(m.arch, 1, BLOCK, "cpu", torch.float32))


# ------------------------------------------------------------------------------------------------ cache sizes, trace replay
def test_cache_rows_follow_the_runs_of_the_layers():
    a = A.from_stack_config(MIXED)
    kv = PagedKVCache(a, 3, BLOCK, "cpu", torch.float32)
    assert kv.full.numel() == 0 and kv.latent.shape == (2, 3 * BLOCK, 56) and sorted(kv.latent_index) == [3, 6] and kv.tokens.shape == (3 * BLOCK,)
    assert [tuple(t.shape[1:]) for t in kv.spec_kv[1]] == [(2, 32), (2, 24)] and kv.spec_kv[1][0] is not kv.spec_kv[4][0]
    per_token = 2 * 40 + 2 * (2 * 56 + 3 * 40 + 56) + 3 * 56
    assert PagedKVCache.bytes_per_block(a, BLOCK, torch.float32) == (per_token * 4 + 4) * BLOCK
    kv.tokens[BLOCK:2 * BLOCK] = 9
    kv.copy_blocks(torch.tensor([1]), torch.tensor([2]))
    assert (kv.tokens[2 * BLOCK:] == 9).all() and (kv.tokens[:BLOCK] == 0).all()
    assert PagedKVCache(A.from_stack_config(dict(MIXED, embedding=dict(scale=1.0))), 3, BLOCK, "cpu", torch.float32).tokens is None


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
