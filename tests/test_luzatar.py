"""Luzatar stacks (gated delta rule and windowed latent attention in parallel blocks on an fp32 residual stream) against the plain
restatement of tests/stack_oracle.py: every mechanism alone, whole models through the engine's step function in all the ways a sequence
can be cut up and batched, and generation through the public entry points.  The CPU cases run the fp32 restatements of the device ops,
the GPU cases the kernels in fp32 and bf16."""
import json
import math

import numpy as np
import pytest
import torch

import onnxruntime_genai_b200 as og
from onnxruntime_genai_b200 import ops
from onnxruntime_genai_b200.models import arch as A
from onnxruntime_genai_b200.models.decoder import PagedKVCache
from stack_harness import BLOCK, RUNTIMES, beam_search, close, dtype_of, feed, greedy_ok, one_thread, open_engine, open_model, paged, random_tokens, rows_of, tol_of  # noqa: F401
from stack_models import delta, latent, stack, weights, write
from stack_oracle import causal_conv_silu, delta_recurrence, layer_norm, rms_norm, rotary_frequencies, rotate, stack_forward, unit_vectors, visible

@pytest.fixture(params=RUNTIMES)
def runtime(request):
    return request.param


# ------------------------------------------------------------------------------------------------ models and engines
MIXED = stack([delta(), latent(scale=0.5), latent(heads=5, window=7, scaled=False, ff=0, scale=0.6), delta(weights_of=0),
               delta(heads=2, kv_heads=1, dim=8, vdim=40, conv=2, ff=0), latent(weights_of=1, scale=0.5)])
# sizes the vector paths cannot take: odd widths, ranks and head sizes, one tap, one head, equal sizes everywhere
ODD = stack([latent(heads=1, dim=9, rot_dim=6, vdim=5, kv_rank=11, window=3, ff=13, scale=0.8), delta(heads=3, kv_heads=3, dim=7, vdim=5, conv=1, ff=0),
             delta(heads=1, kv_heads=1, dim=3, vdim=7, conv=6, ff=21)], vocab=37, width=45, eps=2e-2)
# sizes that take the tensor-core and warp-MMA kernels of both attention forms, every kernel instantiation class of the recurrence
WIDE = stack([latent(heads=4, dim=56, rot_dim=24, vdim=64, kv_rank=88, window=50, ff=128, scale=0.25), delta(heads=4, kv_heads=2, dim=64, vdim=48, ff=192),
              latent(heads=9, dim=104, rot_dim=32, vdim=80, kv_rank=200, window=130, ff=64, scale=0.2, original=64),
              latent(heads=3, dim=136, rot_dim=64, vdim=128, kv_rank=384, window=33, ff=0, scale=0.2), delta(heads=2, kv_heads=1, dim=128, vdim=64, ff=64)],
             vocab=160, width=128)
STACKS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}
# ------------------------------------------------------------------------------------------------ configuration
def test_config_is_read_into_layer_specs():
    a = A.from_stack_config(MIXED)
    assert a.model_type == "luzatar" and a.num_layers == 6 and a.layernorm and a.parallel_block and a.activation == "relu"
    assert a.layer_types == ["linear_attention", "latent_attention", "latent_attention", "linear_attention", "linear_attention", "latent_attention"]
    assert a.layer_specs[1].window == 20 and a.layer_specs[2].ff == 0 and a.layer_specs[2].rotary.scaling is None and a.layer_specs[3].weights_of == 0
    assert a.norm_eps == 3e-5 and a.has_linear_layers
    shapes = A.stack_weight_shapes(a)
    assert "l3.norm1" not in shapes and "l5.mix.q" not in shapes and shapes["l4.mix.v.conv"] == (80, 2) and "l2.mlp.gate" not in shapes


@pytest.mark.parametrize("broken", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][3].update(weights_of=1),
                                    lambda c: c["layers"][0]["mlp"].update(kind="routed"), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10)])
def test_unknown_configurations_are_refused(broken):
    c = json.loads(json.dumps(MIXED))
    broken(c)
    with pytest.raises(ValueError):
        A.from_stack_config(c)


def test_wrong_and_missing_tensors_are_refused(tmp_path):
    w = weights(ODD)
    w["head"] = w["head"][:, :-1]
    with pytest.raises(ValueError, match="head"):
        og.Model(og.Config(write(ODD, w, tmp_path / "a"), provider="cpu"))
    w = weights(ODD)
    del w["l1.mix.a"]
    with pytest.raises(ValueError, match="l1.mix.a"):
        og.Model(og.Config(write(ODD, w, tmp_path / "b"), provider="cpu"))


def test_builder_exports_a_model_directory(tmp_path):
    from onnxruntime_genai_b200.models.builder import main
    d = write(ODD, weights(ODD, 3), tmp_path / "in")
    main(["-m", d, "-o", str(tmp_path / "out"), "-p", "bf16", "-e", "cpu", "--extra_options", "max_batch_size=3"])
    m = og.Model(str(tmp_path / "out"))
    assert m.type == "luzatar" and m.device_type == "cpu" and m.config.engine["dynamic_batching"]["max_batch_size"] == 3
    toks = random_tokens(ODD, 9)
    close(feed(open_engine(m), m, toks, [9]), stack_forward(ODD, weights(ODD, 3), toks)[0], 2e-4)
    main(["-m", d, "-o", str(tmp_path / "syn"), "-p", "fp32", "-e", "cpu", "--extra_options", "synthetic_weights=1", "seed=5"])
    og.Model(str(tmp_path / "syn"))


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("rot", [dict(dims=8, base=5000.0), dict(dims=16, base=100.0, scaling=dict(factor=4.0, original=64, fast=4.0, slow=1.0)),
                                 dict(dims=6, base=10000.0, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                                 dict(dims=12, base=50.0, scaling=dict(factor=2.0, original=100000, fast=2.0, slow=0.5))])
def test_rotary_tables(rot):
    f, amp = rotary_frequencies(rot)
    cos, sin = A.rotary_tables(A.RotarySpec(rot["dims"], rot["base"], rot.get("scaling")), 300)
    for p in (0, 1, 17, 299):
        for i, fi in enumerate(f):
            assert cos[p, i] == pytest.approx(math.cos(p * fi) * amp, abs=1e-6) and sin[p, i] == pytest.approx(math.sin(p * fi) * amp, abs=1e-6)


@pytest.mark.parametrize("H", [24, 45, 512])
def test_stream_norm_and_embedding(runtime, H):
    g = torch.Generator().manual_seed(H)
    x, w, b = torch.randn(7, H, generator=g) * 3 + 2, torch.randn(H, generator=g), torch.randn(H, generator=g)
    dev, dt = runtime[0], dtype_of(runtime)
    rows = torch.tensor([6, 0, 3], dtype=torch.int32)
    want = layer_norm(x.double(), w.double(), b.double(), 0.5)
    close(ops.norm_stream(x.to(dev), w.to(dev), 0.5, b.to(dev), True, dt), want, tol_of(runtime) / 4)
    close(ops.norm_stream(x.to(dev), w.to(dev), 0.5, b.to(dev), True, dt, rows.to(dev)), want[rows.long()], tol_of(runtime) / 4)
    close(ops.norm_stream(x.to(dev), w.to(dev), 0.5, None, False, dt), rms_norm(x.double(), w.double(), 0.5), tol_of(runtime) / 4)
    table = torch.randn(11, H, generator=g).to(dt)
    ids = torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    got = ops.embedding_stream(ids.to(dev), table.to(dev))
    assert got.dtype == torch.float32 and torch.equal(got.cpu(), table[ids.long()].float())


@pytest.mark.parametrize("T,inter,width", [(3, 64, 40), (5, 128, 128), (70, 21, 45), (300, 192, 128)])
def test_relu_gated_feed_forward_into_a_column_range(runtime, T, inter, width):
    g = torch.Generator().manual_seed(T)
    dt, dev = dtype_of(runtime), runtime[0]
    x, w = torch.randn(T, width, generator=g).to(dt), (torch.randn(2 * inter, width, generator=g) / width ** 0.5).to(dt)
    il = runtime == ("cuda", "bfloat16") and inter % 64 == 0
    wide = torch.full((T, inter + 24), 7.0, dtype=dt, device=dev)
    ops.gate_up_act(x.to(dev), (ops.interleave_gate_up(w) if il else w).to(dev), None, "relu", out=wide[:, 8:8 + inter], interleaved=il)
    want = torch.relu(x.double() @ w[:inter].double().T) * (x.double() @ w[inter:].double().T)
    close(wide[:, 8:8 + inter], want, tol_of(runtime))
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + inter:] == 7).all()


@pytest.mark.parametrize("T,K,N", [(1, 40, 72), (6, 45, 37), (64, 256, 512), (500, 128, 200)])
def test_projection_adds_to_the_fp32_stream(runtime, T, K, N):
    g = torch.Generator().manual_seed(K)
    dt, dev = dtype_of(runtime), runtime[0]
    x, w, h = torch.randn(T, K, generator=g).to(dt), torch.randn(N, K, generator=g).to(dt), torch.randn(T, N, generator=g) * 1000
    s = h.to(dev).clone()
    out = ops.linear(x.to(dev), w.to(dev), residual=s, out=s, out_fp32=True)
    assert out.dtype == torch.float32 and out.data_ptr() == s.data_ptr()
    # the stream is not rounded to 16 bits: what was added is exact to fp32 although the stream's values are large
    assert torch.allclose((out.cpu().double() - h.double()), x.double() @ w.double().T, atol=5e-3)


@pytest.mark.parametrize("heads,a_cols,K,N", [(3, 24, 16, 40), (5, 56, 40, 72), (4, 15, 9, 11), (2, 200, 200, 136)])
@pytest.mark.parametrize("T", [1, 20, 130])
def test_per_head_projection(runtime, heads, a_cols, K, N, T):
    g = torch.Generator().manual_seed(N)
    dt, dev = dtype_of(runtime), runtime[0]
    x, w = torch.randn(T, heads * a_cols + 8, generator=g).to(dt), torch.randn(heads * N, K, generator=g).to(dt)
    want = torch.cat([x[:, h * a_cols:h * a_cols + K].double() @ w[h * N:(h + 1) * N].double().T for h in range(heads)], 1)
    close(ops.head_project(x.to(dev), w.to(dev), heads, a_cols), want, tol_of(runtime) / 4)
    wide = torch.zeros(T, heads * N + 16, dtype=dt, device=dev)
    ops.head_project(x.to(dev), w.to(dev), heads, a_cols, out=wide[:, 8:8 + heads * N])
    close(wide[:, 8:8 + heads * N], want, tol_of(runtime) / 4)


@pytest.mark.parametrize("C,L", [(24, 4), (13, 3), (40, 1), (80, 6)])
def test_convolution_continues_over_portions_and_pages(runtime, C, L):
    g = torch.Generator().manual_seed(C)
    dt, dev = dtype_of(runtime), runtime[0]
    seqs = [torch.randn(n, C, generator=g).to(dt) for n in (37, 5, 18)]
    taps = torch.randn(C, L, generator=g).to(dt)
    cache = torch.zeros(12 * BLOCK, C + 3, dtype=dt, device=dev)[:, :C] if C % 8 else torch.zeros(12 * BLOCK, C + 8, dtype=dt, device=dev)[:, :C]
    wide = lambda x: torch.cat([x, x.new_zeros(x.shape[0], (-C) % 8 + 8)], 1)[:, :C]
    got, done = [[] for _ in seqs], [0, 0, 0]
    for cut in ((15, 1, 16), (2, 1, 2), (20, 3, 0)):
        lens = [(d, n) for d, n in zip(done, cut)]
        pg = paged([(d, len(s) - d) for d, s in zip(done, seqs)], 12)       # the same tables in every portion (total length fixed)
        full = paged([(0, len(s)) for s in seqs], 12)
        idx = [i for b, (d, n) in enumerate(lens) for i in range(int(full["cu"][b]) + d, int(full["cu"][b]) + d + n)]
        x = torch.cat([s[d:d + n] for s, (d, n) in zip(seqs, lens)])
        cu = torch.tensor(np.cumsum([0] + list(cut)), dtype=torch.int32)
        y = ops.causal_conv(wide(x).to(dev), taps.to(dev), None, cache, full["slots"][idx].to(dev), full["pos"][idx].to(dev), cu.to(dev),
                            torch.tensor(done, dtype=torch.int32, device=dev), full["table"].to(dev), BLOCK, silu=True)
        for b, n in enumerate(cut):
            got[b].append(y[int(cu[b]):int(cu[b + 1])].cpu())
            done[b] += n
        del pg
    for s, y in zip(seqs, got):
        close(torch.cat(y), causal_conv_silu(s.double(), taps.double()), tol_of(runtime))


@pytest.mark.gpu
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hk,Hv,dk,dv", [(2, 4, 24, 16), (1, 3, 7, 5), (2, 2, 64, 100), (1, 2, 128, 128), (1, 1, 200, 33), (1, 2, 300, 32), (1, 1, 600, 8)])
def test_delta_recurrence_kernels(dt, Hk, Hv, dk, dv):
    """Portions of several sizes and single tokens, requests of unequal length side by side, slots in any order and used again."""
    g = torch.Generator().manual_seed(dk)
    cd, vd, T = 2 * Hk * dk + Hv * dv, Hv * dv, 45
    na, dtb, nw = -torch.exp(torch.randn(Hv, generator=g) - 1), torch.randn(Hv, generator=g) * 0.3, 1 + 0.2 * torch.randn(dv, generator=g)
    stride = Hv * dk * dv + 4
    state = torch.full((5, stride), 99.0, device="cuda")
    view = state[:, :Hv * dk * dv].view(5, Hv, dk, dv)

    def oracle(conv, proj):
        conv, proj = conv.double(), proj.double()
        q, k = (unit_vectors(conv[:, i * Hk * dk:(i + 1) * Hk * dk].view(-1, Hk, dk)) for i in (0, 1))
        a, b, z = proj[:, cd + vd + Hv:], proj[:, cd + vd:cd + vd + Hv], proj[:, cd:cd + vd].view(-1, Hv, dv)
        gate = torch.exp(na.double() * torch.nn.functional.softplus(a + dtb.double()))
        o = delta_recurrence(q * dk ** -0.5, k, conv[:, 2 * Hk * dk:].view(-1, Hv, dv), gate, torch.sigmoid(b))
        return (rms_norm(o, nw.double(), 1e-3) * torch.nn.functional.silu(z)).reshape(-1, vd)

    for rep in range(2):                                   # the second pass reuses the slots: stale states must not leak in
        seqs = [(torch.randn(n, cd, generator=g).to(dt), torch.randn(n, cd + vd + 2 * Hv, generator=g).to(dt)) for n in (T, 9, 33)]
        slots, done, got = torch.tensor([3, 0, 4], dtype=torch.int32, device="cuda"), [0, 0, 0], [[], [], []]
        for cut in ((40, 2, 31), (1, 1, 1), (1, 0, 1), (3, 6, 0)):
            conv = torch.cat([c[d:d + n] for (c, _), d, n in zip(seqs, done, cut)]).cuda()
            proj = torch.cat([p[d:d + n] for (_, p), d, n in zip(seqs, done, cut)]).cuda()
            cu = torch.tensor(np.cumsum([0] + list(cut)), dtype=torch.int32, device="cuda")
            y = ops.gated_delta_layer(conv, proj, cd, vd, Hk, Hv, dk, dv, na.cuda(), dtb.cuda(), nw.cuda(), 1e-3, view, slots, cu,
                                      torch.tensor(done, dtype=torch.int32, device="cuda"), max(cut), 1e-6)
            for b, n in enumerate(cut):
                got[b].append(y[int(cu[b]):int(cu[b + 1])].cpu())
                done[b] += n
        for (c, p), y in zip(seqs, got):
            y = torch.cat(y)
            close(y, oracle(c[:len(y)], p[:len(y)]), 4e-2 if dt == torch.bfloat16 else 2e-4)
    assert (state[:, Hv * dk * dv:] == 99).all() and (state[1] == 99).all() and (state[2] == 99).all()


SHAPES = [(3, 40, 8, 24, 48, 8), (1, 9, 6, 5, 11, 6), (5, 80, 24, 56, 112, 24), (17, 24, 32, 16, 256, 20), (4, 128, 64, 128, 512, 64), (40, 16, 8, 16, 40, 0)]


def _latent_case(shape, lens, window, seed, dt, needles=()):
    """Random projections and a paged cache for requests (past, new); needles (request, position, query position): the key at the
    position is scaled to stand out for that query.  Returns device inputs and the plain result of every new token."""
    H, d, r, dv, R, rd = shape
    g = torch.Generator().manual_seed(seed)
    total = [p + n for p, n in lens]
    rot = dict(dims=rd, base=300.0, scaling=dict(factor=4.0, original=40, fast=6.0, slow=1.0)) if rd else None
    uk, uv, nw = torch.randn(H * d, R, generator=g) / R ** 0.5, torch.randn(H * dv, R, generator=g) / R ** 0.5, 1 + 0.2 * torch.randn(R, generator=g)
    uk, uv = uk.to(dt), uv.to(dt)
    seqs = []
    for b, n in enumerate(total):
        x = torch.randn(n, H * (d + r) + R + r, generator=g)
        for nb, key, query in needles:
            if nb == b:
                # the query's heads point along the key's expanded direction
                c = x[key, H * (d + r):H * (d + r) + R]
                c = c / c.pow(2).mean().sqrt() * nw
                x[query, :H * (d + r)].view(H, d + r)[:, :d] = 6 * (uk.float() @ c).view(H, d) / (uk.float() @ c).view(H, d).norm(dim=-1, keepdim=True) * d ** 0.25
        seqs.append(x.to(dt))
    scale = 1.0 / d ** 0.5
    want = []
    for x, (p, n) in zip(seqs, lens):
        x = x.double()
        T = x.shape[0]
        q, c, kr = x[:, :H * (d + r)].view(T, H, d + r), rms_norm(x[:, H * (d + r):H * (d + r) + R], nw.double(), 1e-5), x[:, H * (d + r) + R:]
        qr, kr = rotate(q[:, :, d:], rot), rotate(kr.view(T, 1, r), rot)[:, 0]
        kn, v = (c @ uk.double().T).view(T, H, d), (c @ uv.double().T).view(T, H, dv)
        s = (torch.einsum("qhd,khd->hqk", q[:, :, :d], kn) + torch.einsum("qhr,kr->hqk", qr, kr)) * scale
        s = s.masked_fill(~visible(T, dict(size=window) if window else None)[None], -math.inf)
        want.append(torch.einsum("hqk,khd->qhd", torch.softmax(s, -1), v).reshape(T, H * dv)[p:])
    return dict(seqs=seqs, uk=uk, uv=uv, nw=nw, rot=rot, scale=scale, want=torch.cat(want))


def _run_latent(case, shape, lens, window, runtime, splits=None, long_tokens=None):
    H, d, r, dv, R, rd = shape
    dev, dt = runtime[0], dtype_of(runtime)
    sh = ops.latent_shape(H, d, r, dv, R, rd)
    pg = paged(lens, sum((p + n + BLOCK - 1) // BLOCK for p, n in lens) + 2, seed=5)
    ld = (R + r + 7) // 8 * 8 + 8
    cache = torch.full(((int(pg["table"].max()) + 3) * BLOCK, ld), 3.0, dtype=dt, device=dev)
    cos = sin = None
    if rd:
        cos, sin = (torch.from_numpy(t).to(dev) for t in A.rotary_tables(A.RotarySpec(rd, case["rot"]["base"], case["rot"]["scaling"]), 2048))
    wide = lambda x: torch.cat([x, x.new_zeros(x.shape[0], (-x.shape[1]) % 8)], 1).to(dev)[:, :x.shape[1]]
    N = H * (d + r) + R + r
    for b, (p, n) in enumerate(lens):            # what earlier steps left in the cache
        if p:
            ops.latent_prep(wide(case["seqs"][b][:p].clone()), sh, case["nw"].to(dev), 1e-5, torch.arange(p, dtype=torch.int32, device=dev), cos, sin,
                            rows_of(pg, b, p).to(torch.int32).to(dev), cache)
    proj = wide(torch.cat([s[p:] for s, (p, _) in zip(case["seqs"], lens)]).clone())
    t = {k: v.to(dev) for k, v in pg.items()}
    ops.latent_prep(proj, sh, case["nw"].to(dev), 1e-5, t["pos"], cos, sin, t["slots"], cache)
    assert proj.shape[1] == N and (cache[:, R + r:] == 3).all()
    out = torch.zeros(proj.shape[0], H * dv, dtype=dt, device=dev)
    uk_t = case["uk"].view(H, d, R).transpose(1, 2).reshape(H * R, d).contiguous().to(dev)
    mq, mk = max(n for _, n in lens), max(p + n for p, n in lens)
    plan = ops.LatentPlan(lens, window, dev, long_tokens) if long_tokens is not None else None
    if long_tokens is None or any(n < long_tokens for _, n in lens):
        qlat = ops.head_project(proj, uk_t, H, d + r)
        olat = ops.latent_attention(qlat, proj, sh, cache, t["cu"], t["past"], t["table"], BLOCK, case["scale"], window, mq, mk,
                                    skip_q_len=long_tokens or 0, splits=splits)
        ops.head_project(olat, case["uv"].to(dev), H, R, out=out)
    if plan is not None and plan.rows:
        assert ops.latent_long_supported(sh, proj, cache, BLOCK)
        ops.latent_attention_long(proj, sh, torch.cat([case["uk"], case["uv"]]).to(dev), cache, plan, t["cu"], t["past"], t["table"], BLOCK, case["scale"],
                                  window, out)
    if dev == "cuda":
        ops.check_kernel_status()
    return out


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [0, 1, 23])
def test_latent_attention_over_pages(runtime, shape, window):
    for lens in ([(0, 1), (70, 1), (15, 1), (16, 1), (200, 1)], [(0, 5), (31, 2), (40, 33), (17, 1)]):
        case = _latent_case(shape, lens, window, 3, dtype_of(runtime))
        for splits in (None, 1, 3):
            close(_run_latent(case, shape, lens, window, runtime, splits), case["want"], tol_of(runtime))


@pytest.mark.gpu
@pytest.mark.parametrize("shape", [(2, 64, 24, 64, 144, 24), (3, 40, 8, 24, 48, 8), (2, 128, 64, 128, 256, 64), (2, 72, 32, 104, 136, 32), (2, 192, 64, 128, 512, 64),
                                   (2, 136, 8, 56, 64, 8)], ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [0, 1, 33, 200])
def test_latent_attention_of_long_prompts_on_expanded_keys(shape, window):
    rt = ("cuda", "bfloat16")
    for lens in ([(0, 300)], [(5, 1), (131, 140), (0, 3), (400, 129), (17, 64)]):
        case = _latent_case(shape, lens, window, 4, torch.bfloat16)
        close(_run_latent(case, shape, lens, window, rt, long_tokens=16), case["want"], tol_of(rt))


@pytest.mark.parametrize("window", [17, 32, 50])
@pytest.mark.parametrize("form", ["decode", "portion", "long"])
def test_window_edges_with_keys_that_stand_out(runtime, window, form):
    """One key dominates its query's scores: just inside the window it decides the result, one position further out it must not count;
    the same for the sequence's first tokens and at page borders."""
    if form == "long" and runtime != ("cuda", "bfloat16"):
        pytest.skip("the expanded form exists in bf16 on the GPU")
    shape = (2, 56, 24, 64, 120, 24)
    for q in (window - 1, window, 64, 79, 80, 127):
        for dist in (0, 1, window - 1, window, window + 1):
            key = q - dist
            if key < 0:
                continue
            n = {"decode": 1, "portion": 7, "long": min(q + 1, 70)}[form]
            lens = [(max(0, q + 1 - n), min(n, q + 1)), (3, 2)]
            case = _latent_case(shape, lens, window, 11 + q + dist, dtype_of(runtime), needles=[(0, key, q)])
            got = _run_latent(case, shape, lens, window, runtime, long_tokens=16 if form == "long" else None)
            close(got, case["want"], tol_of(runtime))


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", list(STACKS))
def test_logits_of_a_whole_prompt(tmp_path_factory, runtime, name):
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    for n in (1, 2, 47, 150):
        toks = random_tokens(cfg, n, n)
        close(feed(open_engine(m), m, toks, [n]), stack_forward(cfg, w, toks)[0], tol_of(runtime))


@pytest.mark.parametrize("name", list(STACKS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2, 2, 17, 1, 1, 40], [100, 1], [64, 63, 2, 1], [15, 1, 1, 1, 16, 33]], ids=str)
def test_portions_and_single_tokens(tmp_path_factory, runtime, name, cuts):
    """The same logits whatever the cut: token by token, pairs, ends and starts of pages and windows, long portions then decoding."""
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    toks = random_tokens(cfg, 130, 7)
    close(feed(open_engine(m), m, toks, cuts), stack_forward(cfg, w, toks)[0], tol_of(runtime))


@pytest.mark.parametrize("name", list(STACKS))
def test_mixed_batches_reuse_pages_and_slots(tmp_path_factory, runtime, name):
    """More requests than fit at once come and go through a pool that is just large enough, portions beside single tokens, requests left
    out of some steps; every request gets the logits it gets alone."""
    m, cfg, w = open_model(tmp_path_factory, name, runtime, STACKS[name])
    eng = open_engine(m, blocks=26, batch=4, tokens=300)
    rng = np.random.RandomState(5)
    waiting = [(i, random_tokens(cfg, n, 20 + i)) for i, n in enumerate((90, 33, 120, 5, 64, 1, 77, 100, 16, 50))]
    live, got, seen = [], {i: [] for i, _ in waiting}, dict(waiting)
    used_blocks = set()
    while waiting or live:
        while waiting and len(live) < 4 and sum((len(t) + BLOCK - 1) // BLOCK for _, t, _, _ in live) + (len(waiting[0][1]) + BLOCK - 1) // BLOCK <= 26:
            i, t = waiting.pop(0)
            live.append([i, t, 0, og.Request(og.GeneratorParams(m))])
        step = []
        for e in live:
            if len(live) > 1 and rng.rand() < 0.25:
                continue                                    # left out of this step
            n = min(int(rng.choice([1, 1, 2, 3, 17, 40, 70])), len(e[1]) - e[2])
            step.append((e, n))
        if not step:
            continue
        out = eng.run_given([(e[3], e[1][e[2]:e[2] + n], list(range(n)) if e[0] % 2 else [n - 1]) for e, n in step])
        eng.core.check_invariants()
        for (e, n), lg in zip(step, out):
            got[e[0]].append((e[2], n, lg.float().cpu()))
            e[2] += n
            used_blocks.update(e[3]._native.blocks())
        for e in [e for e in live if e[2] == len(e[1])]:
            eng.remove_request(e[3])
            live.remove(e)
    assert eng.core.free_blocks == 26 and len(eng._free_slots) == 4
    for i, parts in got.items():
        want = stack_forward(cfg, w, seen[i])[0]
        for at, n, lg in parts:
            close(lg, want[at:at + n] if i % 2 else want[at + n - 1:at + n], 1.5 * tol_of(runtime))


def test_a_request_does_not_see_the_batch_around_it(tmp_path_factory, runtime):
    m, cfg, _ = open_model(tmp_path_factory, "wide", runtime, STACKS["wide"])
    a, b, c = (random_tokens(cfg, n, s) for n, s in ((90, 1), (75, 2), (3, 3)))
    alone = feed(open_engine(m), m, a, [80, 1])
    eng = open_engine(m)
    ra, rb, rc = (og.Request(og.GeneratorParams(m)) for _ in range(3))
    rows = [eng.run_given([(rb, b[:70], []), (ra, a[:80], list(range(80))), (rc, c, [0])])[1]]
    for j in range(10):
        rows.append(eng.run_given([(ra, a[80 + j:81 + j], [0])] + ([(rb, b[70 + j:71 + j], [0])] if j < 5 else []))[0])
    close(torch.cat(rows), alone.double(), tol_of(runtime) / 4)


def test_long_decoding(tmp_path_factory, runtime):
    """Hundreds of single-token steps: windows slide over decoded tokens, states are carried on, pages fill up."""
    m, cfg, w = open_model(tmp_path_factory, "mixed", runtime, STACKS["mixed"])
    toks = random_tokens(cfg, 260, 9)
    close(feed(open_engine(m), m, toks, [20, 1]), stack_forward(cfg, w, toks)[0], tol_of(runtime))


def test_run_given_rejects_what_does_not_fit(tmp_path_factory):
    m, cfg, _ = open_model(tmp_path_factory, "odd", ("cpu", "float32"), STACKS["odd"])
    eng = open_engine(m, blocks=4, batch=2, tokens=64)
    r = og.Request(og.GeneratorParams(m))
    with pytest.raises(RuntimeError):
        eng.run_given([(r, random_tokens(cfg, 3), [3])])
    with pytest.raises(RuntimeError):
        eng.run_given([(og.Request(og.GeneratorParams(m)), random_tokens(cfg, 65), [])])


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_through_generator_and_engine(tmp_path_factory, runtime):
    m, cfg, w = open_model(tmp_path_factory, "wide", runtime, STACKS["wide"])
    tol = 0.2 if runtime[1] == "bfloat16" else 1e-3
    prompts = [random_tokens(cfg, n, 40 + n) for n in (70, 5, 33, 1, 18)]
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=100, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompts[0].astype(np.int32).reshape(1, -1))
    while not gen.is_done():
        gen.generate_next_token()
    solo = np.asarray(gen.get_sequence(0))[70:]
    assert len(solo) == 30
    greedy_ok(cfg, w, prompts[0], solo, tol)
    # the scheduler: more requests than the batch holds, prompts cut by a small token budget, blocks that run short
    eng = open_engine(m, blocks=30, batch=3, tokens=40)
    reqs = []
    for t in prompts:
        gp = og.GeneratorParams(m)
        gp.set_search_options(max_length=len(t) + 25, do_sample=False)
        r = og.Request(gp)
        r.add_tokens(t.astype(np.int32))
        eng.add_request(r)
        reqs.append(r)
    while eng.has_pending_requests():
        r = eng.step()
        if r is None:
            continue
        while r.has_unseen_tokens():
            r.get_unseen_token()
        if r.is_turn_complete():
            r.kept = r.tokens()
            eng.remove_request(r)
    for r, t in zip(reqs, prompts):
        assert len(r.kept) == len(t) + 25
        greedy_ok(cfg, w, t, r.kept[len(t):], tol)


def test_batched_generator_rewind_and_beams(tmp_path_factory, runtime):
    m, cfg, w = open_model(tmp_path_factory, "mixed", runtime, STACKS["mixed"])
    tol = 0.2 if runtime[1] == "bfloat16" else 1e-3
    prompt = np.stack([random_tokens(cfg, 12, 3), random_tokens(cfg, 12, 4)]).astype(np.int32)
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=30, batch_size=2, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt)
    while not gen.is_done():
        gen.generate_next_token()
    for r in range(2):
        greedy_ok(cfg, w, prompt[r], np.asarray(gen.get_sequence(r))[12:], tol)
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=40, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt[:1])
    for _ in range(10):
        gen.generate_next_token()
    first = np.asarray(gen.get_sequence(0)).copy()
    gen.rewind_to(15)
    for _ in range(7):
        gen.generate_next_token()
    greedy_ok(cfg, w, prompt[0], np.asarray(gen.get_sequence(0))[12:], tol)
    assert (np.asarray(gen.get_sequence(0))[:15] == first[:15]).all()
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=24, num_beams=3, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt[:1])
    while not gen.is_done():
        gen.generate_next_token()
    seq = np.asarray(gen.get_sequence(0))
    lp = lambda s: float(sum(torch.log_softmax(stack_forward(cfg, w, s)[0], -1)[i, int(s[i + 1])] for i in range(11, len(s) - 1)))
    # beams follow their own states and pages: a plain beam search over the restatement finds a hypothesis of the same score (16-bit
    # rounding may pick another one where candidates are close)
    best = lp(beam_search(cfg, w, prompt[0], 24, 3))
    assert abs(lp(seq) - best) < (4.0 if runtime[1] == "bfloat16" else 2e-2)


# ------------------------------------------------------------------------------------------------ cache sizes, trace replay
def test_cache_rows_follow_the_layers():
    a = A.from_stack_config(MIXED)
    kv = PagedKVCache(a, 3, BLOCK, "cpu", torch.float32)
    assert kv.full.numel() == 0 and kv.latent.shape == (3, 3 * BLOCK, 56) and kv.conv.shape == (3, 3 * BLOCK, 160)
    assert kv.conv_layer(4).shape == (3 * BLOCK, 96) and kv.conv_layer(0).shape == (3 * BLOCK, 160)
    kv.ensure_state_slots(2)
    assert kv.state.shape == (3, 2, 1536) and kv.state_layer(4).shape == (2, 2, 8, 40)
    assert PagedKVCache.bytes_per_block(a, BLOCK, torch.float32) == (3 * 56 + 3 * 160) * 4 * BLOCK


def test_trace_replay_writes_the_wanted_rows(tmp_path):
    from onnxruntime_genai_b200 import trace_replay
    cfg, w = ODD, weights(ODD, 8)
    c = og.Config(write(cfg, w, tmp_path / "m"), provider="cpu")
    m = og.Model(c)
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
