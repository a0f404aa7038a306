"""A slow, plain restatement of declared-stack decoders (gated-delta and latent-attention mixers in parallel blocks; chunked attention
with sinks and routed experts in blocks whose norms follow the sub-layers; soft-capped, differential and query-compressed latent attention with
output gates in pre-norm blocks that run several times; attention with mixed heads beside a gated recurrence, and matrix memories, in parallel blocks
with a norm per sub-layer), one function per mechanism, token by token where the mechanism is a recurrence.  It shares no code with the package: the tests compare the
runtime against it.  Weights come as a dictionary of tensors under the checkpoint's names; all math runs in `dtype` (float64 by
default).  A whole sequence is evaluated at once, from its first token: there is no cache here."""
import math

import torch


# ------------------------------------------------------------------------------------------------ mechanisms
def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def causal_conv_silu(x, taps):
    """x [T, C], taps [C, K]: the newest position meets the last column."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for k in range(K):
            if t - k >= 0:
                y[t] = y[t] + taps[:, K - 1 - k] * x[t - k]
    return y * torch.sigmoid(y)


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta):
    """q, k [T, Hk, dk] (prepared), v [T, H, dv], decay g and strength beta [T, H] -> [T, H, dv]."""
    T, H, dv = v.shape
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], dv, dtype=v.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = S[h] * g[t, h]
            u = beta[t, h] * (v[t, h] - kk @ S[h])
            S[h] = S[h] + torch.outer(kk, u)
            out[t, h] = qq @ S[h]
    return out


def delta_mixer(x, w, p, m, eps):
    """x [T, width]; w: weights, p: prefix of the layer's mixer tensors, m: the mixer's sizes."""
    T, H, Hk, dk, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv_silu(x @ w[p + "q"].T, w[p + "q.conv"]).view(T, Hk, dk)
    k = causal_conv_silu(x @ w[p + "k"].T, w[p + "k.conv"]).view(T, Hk, dk)
    v = causal_conv_silu(x @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, dv)
    q, k = unit_vectors(q) * dk ** -0.5, unit_vectors(k)
    beta = torch.sigmoid(x @ w[p + "b"].T)
    step = torch.log1p(torch.exp(-(x @ w[p + "a"].T + w[p + "dt_bias"]).abs())) + (x @ w[p + "a"].T + w[p + "dt_bias"]).clamp(min=0)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * step)
    o = delta_recurrence(q, k, v, g, beta)
    z = (x @ w[p + "g"].T).view(T, H, dv)
    o = rms_norm(o, w[p + "norm"], eps) * (z * torch.sigmoid(z))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def wavelength_scaled(f, s):
    """Frequency f slowed down by s["factor"] where its wavelength is long against the original context, kept where it is short, blended
    between."""
    wave = 2 * math.pi / f
    if wave < s["original"] / s["high"]:
        return f
    if wave > s["original"] / s["low"]:
        return f / s["factor"]
    keep = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
    return keep * f + (1 - keep) * f / s["factor"]


def rotary_frequencies(rot):
    """(frequency of every pair, factor on cos and sin)."""
    d, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / d) for i in range(d // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    if "low" in s:
        return [wavelength_scaled(fi, s) for fi in f], 1.0
    if "original" not in s:
        return [fi / s["factor"] for fi in f], 1.0

    def turns(t):
        return d * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), d - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, >= dims]: pairs (i, i + dims / 2) of the first dims entries turn with the position."""
    if not rot:
        return x
    f, amp = rotary_frequencies(rot)
    half = rot["dims"] // 2
    y, pos = x.clone(), torch.arange(x.shape[0], dtype=torch.float64)[:, None]
    for i in range(half):
        c, s = (torch.cos(pos * f[i]) * amp).to(x.dtype), (torch.sin(pos * f[i]) * amp).to(x.dtype)
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def rotate_neighbours(x, rot):
    """x [T, heads, >= dims]: pairs (2 i, 2 i + 1) of the first dims entries turn with the position."""
    if not rot:
        return x
    f, amp = rotary_frequencies(rot)
    y, pos = x.clone(), torch.arange(x.shape[0], dtype=torch.float64)[:, None]
    for i, fi in enumerate(f):
        c, s = (torch.cos(pos * fi) * amp).to(x.dtype), (torch.sin(pos * fi) * amp).to(x.dtype)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(T, mask):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = j <= i
    if mask:
        ok = ok & (i - j < mask["size"])
    return ok


def latent_mixer(x, w, p, m, eps):
    T, H, d, r, dv, R = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (x @ w[p + "q"].T).view(T, H, d + r)
    down = x @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    kr = rotate(down[:, R:].view(T, 1, r), m.get("rot"))[:, 0]
    qr = rotate(q[:, :, d:], m.get("rot"))
    kn = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    ok = visible(T, m.get("mask"))
    out = torch.zeros(T, H, dv, dtype=x.dtype)
    for h in range(H):
        s = (q[:, h, :d] @ kn[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        out[:, h] = torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v[:, h]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def same_chunk(T, size):
    """ok[i, j]: j is not after i and in the same run of `size` positions (runs are counted from position 0)."""
    ok = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        ok[i, i // size * size:i + 1] = True
    return ok


def sink_attention(q, k, v, ok, scale, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; sink [H]: a logit in the denominator that has no key and no value."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~ok, -math.inf)
        top = torch.maximum(s.max(-1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = (e @ v[:, g]) / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - top))
    return out


def attention_mixer(x, w, p, m, eps):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((x @ w[p + "q"].T).view(T, H, d), w[p + "q.norm"], eps)
    k = rms_norm((x @ w[p + "k"].T).view(T, G, d), w[p + "k.norm"], eps)
    v = (x @ w[p + "v"].T).view(T, G, dv)
    q, k = rotate(q, m.get("rot")), rotate(k, m.get("rot"))
    o = sink_attention(q, k, v, same_chunk(T, m["mask"]["size"]), m["scale"], w[p + "sink"])
    o = o * torch.sigmoid(x @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_feed_forward(x, w, p, m=None):
    return (gelu_tanh(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(x, w, p, limit):
    g, u = (x @ w[p + "gate"].T).clamp(max=limit), (x @ w[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def routed_experts(x, w, p, m):
    """Each token: the `top` experts of largest probability, weighted by their probabilities among all experts."""
    s = torch.softmax(x @ w[p + "router"].T, -1)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in torch.argsort(s[t], descending=True)[:m["router"]["top"]].tolist():
            out[t] = out[t] + s[t, e] * clamped_expert(x[t:t + 1], w, f"{p}e{e}.", m["expert"]["limit"])[0]
    return out


def feed_forward(x, w, p):
    return (torch.relu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def bounded_norm(x, w, p):
    """Norm without statistics: a scaled hyperbolic tangent of every entry, weight and bias."""
    return torch.tanh(w[p + ".alpha"] * x) * w[p] + w[p + ".b"]


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of every token in a table over hashed pairs (previous token, token); a first token has the row behind the buckets."""
    return [buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tokens[t]) * mul_cur) % buckets for t in range(len(tokens))]


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def softmax_attention(q, k, v, ok, scale, cap=0.0):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    rep = q.shape[1] // k.shape[1]
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=q.dtype)
    for h in range(q.shape[1]):
        s = capped(q[:, h] @ k[:, h // rep].T * scale, cap)
        out[:, h] = torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v[:, h // rep]
    return out


def gated_output(o, x, w, p):
    """Concatenated heads, element by element times the sigmoid of a projection of the mixer's input; output map."""
    return (o.reshape(o.shape[0], -1) * torch.sigmoid(x @ w[p + "g"].T)) @ w[p + "o"].T


def capped_mixer(x, w, p, m, eps):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((x @ w[p + n].T + w[p + n + ".b"]).view(T, h, c) for n, h, c in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = rotate_neighbours(q, m.get("rot")), rotate_neighbours(k, m.get("rot"))
    return gated_output(softmax_attention(q, k, v, visible(T, m.get("mask")), m["scale"], m.get("softcap")), x, w, p)


def difference_factor(w, p, diff):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def difference_of_maps(a1, a2, factor, diff, eps):
    """a1, a2 [T, H, dv]: what two attention maps make of the same values."""
    o = a1 - factor * a2
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * (1 - diff)


def differential_mixer(x, w, p, m, eps):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ w[p + "q"].T + w[p + "q.b"]).view(T, H, 2, d)
    k = (x @ w[p + "k"].T + w[p + "k.b"]).view(T, G, 2, d)
    v = (x @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    ok = visible(T, m.get("mask"))
    a = [softmax_attention(rotate(q[:, :, i], m.get("rot")), rotate(k[:, :, i], m.get("rot")), v, ok, m["scale"]) for i in (0, 1)]
    return gated_output(difference_of_maps(*a, difference_factor(w, p, m["diff"]), m["diff"], eps), x, w, p)


def compressed_latent_mixer(x, w, p, m, eps):
    """Latent attention whose queries come out of a normed latent of their own, with sinks and an output gate."""
    T, H, d, r, dv, R = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(x @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d + r)
    down = x @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    kr = rotate(down[:, R:].view(T, 1, r), m.get("rot"))
    q = torch.cat([q[:, :, :d], rotate(q[:, :, d:], m.get("rot"))], -1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr.expand(T, H, r)], -1)
    o = sink_attention(q, k, (c @ w[p + "uv"].T).view(T, H, dv), visible(T, m.get("mask")), m["scale"], w[p + "sink"])
    return gated_output(o, x, w, p)


def selected_experts(x, w, p, m):
    """Each token: the `top` experts of largest router logit, weighted by a softmax over these logits; a shared expert for every token."""
    z = x @ w[p + "router"].T
    out = clamped_expert(x, w, p + "shared.", m["shared"]["limit"]) if m.get("shared") else torch.zeros_like(x)
    for t in range(x.shape[0]):
        chosen = torch.argsort(z[t], descending=True)[:m["router"]["top"]]
        for e, share in zip(chosen.tolist(), torch.softmax(z[t, chosen], -1)):
            out[t] = out[t] + share * clamped_expert(x[t:t + 1], w, f"{p}e{e}.", m["expert"]["limit"])[0]
    return out


def mixed_scores(q, k, mix, scale):
    """Scores [H, T, T] of q [T, H, d] and k [T, G, d], head h a sum of all heads' scores weighted by mix[h]."""
    H, rep = q.shape[1], q.shape[1] // k.shape[1]
    own = torch.stack([q[:, h] @ k[:, h // rep].T * scale for h in range(H)])
    return torch.stack([sum(mix[h, g] * own[g] for g in range(H)) for h in range(H)])


def mixed_heads_attention(q, k, v, ok, scale, mix):
    """q [T, H, d], k [T, G, d], v [T, G, dv], mix [H, H] -> [T, H, dv]."""
    rep = q.shape[1] // k.shape[1]
    s = mixed_scores(q, k, mix, scale)
    return torch.stack([torch.softmax(s[h].masked_fill(~ok, -math.inf), -1) @ v[:, h // rep] for h in range(q.shape[1])], 1)


def mixed_heads_mixer(x, w, p, m, eps):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((x @ w[p + n].T + w[p + n + ".b"]).view(T, h, c) for n, h, c in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = (rotate(rms_norm(t, w[p + n + ".norm"], eps), m.get("rot")) for t, n in ((q, "q"), (k, "k")))
    o = mixed_heads_attention(q, k, v, visible(T, m.get("mask")), m["scale"], w[p + "talk"])
    return gated_output(o, x, w, p) + w[p + "o.b"]


def gated_average(z, u):
    """S_t = (1 - z_t) S_(t-1) + z_t c(u_t) from S = 0, per column; c(u) = u + 1/2 above zero, sigmoid(u) below."""
    S, out = torch.zeros_like(u[0]), torch.zeros_like(u)
    for t in range(u.shape[0]):
        c = torch.where(u[t] >= 0, u[t] + 0.5, torch.sigmoid(u[t]))
        S = (1 - z[t]) * S + z[t] * c
        out[t] = S
    return out


def gated_average_mixer(x, w, p, m, eps):
    S = gated_average(torch.sigmoid(x @ w[p + "z"].T + w[p + "z.b"]), x @ w[p + "x"].T + w[p + "x.b"])
    g = x @ w[p + "g"].T
    return (S * g * torch.sigmoid(g)) @ w[p + "o"].T


def side_by_side_mixer(x, w, p, m, eps):
    return (m["left_scale"] * mixed_heads_mixer(x, w, p + "left.", m["left"], eps) + m["right_scale"] * gated_average_mixer(x, w, p + "right.", m["right"], eps))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, dv], log gates i (input) and f (forget) [T, H] -> [T, H, dv]; the stored sums are kept relative to exp(m)."""
    T, H, dv = v.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S, n, m = torch.zeros(q.shape[2], dv, dtype=v.dtype), torch.zeros(q.shape[2], dtype=v.dtype), torch.zeros((), dtype=v.dtype)
        for t in range(T):
            new = torch.maximum(f[t, h] + m, i[t, h])
            keep, add = torch.exp(f[t, h] + m - new), torch.exp(i[t, h] - new)
            S, n, m = keep * S + add * torch.outer(k[t, h], v[t, h]), keep * n + add * k[t, h], new
            out[t, h] = (q[t, h] @ S) / (torch.maximum((q[t, h] @ n).abs(), torch.exp(-m)) + 1e-6)
    return out


def matrix_memory_mixer(x, w, p, m, eps):
    T, H, d, dv, cap = x.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k, v = (x @ w[p + "q"].T).view(T, H, d) * d ** -0.5, (x @ w[p + "k"].T).view(T, H, d), (x @ w[p + "v"].T).view(T, H, dv)
    i = capped(x @ w[p + "i"].T + w[p + "i.b"], cap)
    f = -torch.log1p(torch.exp(-capped(x @ w[p + "f"].T + w[p + "f.b"], cap)))
    o = rms_norm(matrix_memory(q, k, v, i, f), 1.0, eps).reshape(T, H * dv) * w[p + "norm"]
    return gated_output(o, x, w, p)


def erf_feed_forward(x, w, p, m=None):
    y = x @ w[p + "up"].T
    return (0.5 * y * (1 + torch.erf(y / math.sqrt(2)))) @ w[p + "down"].T


def squared_relu_expert(x, w, p):
    return torch.relu(x @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def grouped_choice(c, count, keep, top):
    """Indices of the `top` largest of c [E] among the `keep` groups of neighbours whose two largest entries have the largest sums."""
    group = c.view(count, -1)
    best = torch.sort(group, -1, descending=True).values[:, :2].sum(-1)
    open_ = torch.zeros(count, dtype=torch.bool)
    open_[torch.argsort(best, descending=True)[:keep]] = True
    return torch.argsort(group.masked_fill(~open_[:, None], -math.inf).reshape(-1), descending=True)[:top]


def grouped_experts(x, w, p, m):
    """Each token: experts chosen by sigmoid scores plus a correction, weighted by the scores' shares times the router's scale."""
    r = m["router"]
    s = torch.sigmoid(x @ w[p + "router"].T)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        chosen = grouped_choice(s[t] + w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"])
        share = s[t, chosen] / (s[t, chosen].sum() + 1e-20) * r["scale"]
        for e, a in zip(chosen.tolist(), share):
            out[t] = out[t] + a * squared_relu_expert(x[t:t + 1], w, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------------------------------------ the stack
MIXERS = {"delta": delta_mixer, "latent_attention": latent_mixer, "attention": attention_mixer}
FEED_FORWARDS = {"dense": gelu_feed_forward, "moe": routed_experts}


def parallel_block(x, w, p, e, eps, cfg):
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    y = MIXERS[e["type"]](h, w, p + "mix.", e["mixer"], eps)
    if e.get("mlp"):
        y = y + feed_forward(h, w, p + "mlp.")
    return x + y


def output_normed_block(x, w, p, e, eps, cfg):
    """The sub-layers read the stream itself; their results are normed, scaled per element and by the model's multiplier, and added."""
    m = cfg["residual_mult"]
    x = x + m * w[p + "ls1"] * rms_norm(MIXERS[e["type"]](x, w, p + "mix.", e["mixer"], eps), 1 + w[p + "norm1"], eps)
    if e.get("mlp"):
        x = x + m * w[p + "ls2"] * rms_norm(FEED_FORWARDS[e["mlp"]["kind"]](x, w, p + "mlp.", e["mlp"]), 1 + w[p + "norm2"], eps)
    return x


GATED_MIXERS = {"attention": capped_mixer, "attention_2": differential_mixer, "latent_attention": compressed_latent_mixer}


def bounded_norm_block(x, w, p, e, eps):
    x = x + GATED_MIXERS[e["type"]](bounded_norm(x, w, p + "norm1"), w, p + "mix.", e["mixer"], eps)
    if e.get("mlp"):
        x = x + selected_experts(bounded_norm(x, w, p + "norm2"), w, p + "mlp.", e["mlp"])
    return x


def passes(cfg):
    """(layer, pass that starts with it or None) in the order in which the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] + [(i, None) for i in range(b, n)]


def looped_forward(cfg, weights, tokens, dtype=torch.float64):
    """stack_forward of stacks with a hashed-pair embedding, bounded norms and layers that run several times."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    emb = cfg["embedding"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * emb["scale"]
    if emb.get("bigram"):
        x = x + w["bigram"][bigram_rows(tokens, **emb["bigram"])]
    first, streams = x, []
    for i, t in passes(cfg):
        if t is not None:
            x = x + (first if t > 0 else 0) + w["loop.step"][t]
        x = bounded_norm_block(x, w, f"l{i}.", cfg["layers"][i], cfg["norm"]["eps"])
        streams.append(x)
    return bounded_norm(x, w, "final.norm") @ w["head"].T, torch.stack(streams)


TWO_NORM_MIXERS = {"parallel": side_by_side_mixer, "mlstm": matrix_memory_mixer}
TWO_NORM_FEED_FORWARDS = {"dense": erf_feed_forward, "moe": grouped_experts}


def two_norm_parallel_block(x, w, p, e, eps):
    y = TWO_NORM_MIXERS[e["type"]](layer_norm(x, w[p + "norm1"], 0, eps), w, p + "mix.", e["mixer"], eps)
    if e.get("mlp"):
        y = y + TWO_NORM_FEED_FORWARDS[e["mlp"]["kind"]](layer_norm(x, w[p + "norm2"], 0, eps), w, p + "mlp.", e["mlp"])
    return x + y


def two_norm_forward(cfg, weights, tokens, dtype=torch.float64):
    """stack_forward of parallel blocks with a norm per sub-layer."""
    w, eps = {k: v.to(dtype) for k, v in weights.items()}, cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    streams = []
    for i, _ in passes(cfg):
        x = two_norm_parallel_block(x, w, f"l{i}.", cfg["layers"][i], eps)
        streams.append(x)
    return layer_norm(x, w["final.norm"], 0, eps) @ w["head"].T, torch.stack(streams)


def stack_forward(cfg, weights, tokens, dtype=torch.float64):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    if cfg["architecture"] == "Tevilix":
        return two_norm_forward(cfg, weights, tokens, dtype)
    if cfg["architecture"] == "Sugelix":
        return looped_forward(cfg, weights, tokens, dtype)
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg.get("embedding", {}).get("scale", 1.0)
    block = {"Luzatar": parallel_block, "Zevopel": output_normed_block}[cfg["architecture"]]
    streams = []
    for i, e in enumerate(cfg["layers"]):
        p = f"l{e.get('weights_of', i) if e.get('weights_of') is not None else i}."
        x = block(x, w, p, e, eps, cfg)
        streams.append(x)
    if cfg["architecture"] == "Luzatar":
        x = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    else:
        x = rms_norm(x, 1 + w["final.norm"], eps)
    return x @ w["head"].T, torch.stack(streams)
