"""The Gatarax decoder restated plainly: float64 torch on the CPU, whole sequences at once, one function per mechanism,
no cache, no batching, no code shared with the library.  The tests compare the engine with this.

Notation: T tokens, D the stream's width; W["name"] the tensors under the names of the weight file (matrices
[out, in]); t is a query's position and s a key's, both counted from 0.
"""
import math

import torch


# ---- small pieces ---------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The file holds the weight minus one."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def short_conv(u, taps):
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), nothing before the sequence's start."""
    T, C = u.shape
    K = taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(K):
        back = K - 1 - j
        if back < T:
            y[back:] += taps[:, j] * u[:T - back]
    return y


def input_conv(h, taps):
    return h + short_conv(h, taps)


# ---- mixers ---------------------------------------------------------------------------------------------
def sink_weights(scores, visible):
    """softmax whose denominator has one more term exp(0): [H, T, T] scores, [T, T] visibility."""
    scores = scores.masked_fill(~visible[None], float("-inf"))
    top = scores.amax(-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def window_attention(h, W, p, m):
    """Attention without rotation: biased projections, each behind a short convolution, keys limited to the last `size`
    positions, a sink of score 0, a biased output projection."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ W[p + n].T + W[p + n + ".b"], W[p + n + ".conv"]) for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    t = torch.arange(T)
    back = t[:, None] - t[None, :]
    visible = back >= 0
    if m.get("mask") is not None:
        visible = visible & (back < m["mask"]["size"])
    w = sink_weights(torch.einsum("thd,shd->hts", q, k) * m["scale"], visible)
    return torch.einsum("hts,shd->thd", w, v).reshape(T, H * dv) @ W[p + "o"].T + W[p + "o.b"]


def channel_decays(h, W, p, H, d):
    """exp(-exp(A_log_h) softplus(W_a2 (W_a1 h) + dt_bias)): one per head and key channel, [T, H, d]."""
    raw = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    return torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(raw).view(-1, H, d))


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(h, W, p, m, eps):
    """Per head a state S [d, dv];  S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vectors(q.view(T, G, d)) * d ** -0.5
    k = unit_vectors(k.view(T, G, d))
    q, k, v = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1), v.view(T, H, dv)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = channel_decays(h, W, p, H, d)
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    o = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkd,hk->hd", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkd,hk->hd", S, q[t])
    gate = torch.sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, dv)
    return (unit_rms(o, eps) * W[p + "norm"] * gate).reshape(T, H * dv) @ W[p + "o"].T


def side_by_side(h, W, p, m, eps):
    """Half the sum of the two members' results, each RMS-normed over the width first (plain weights)."""
    left = window_attention(h, W, p + "left.", m["left"])
    right = delta_rule(h, W, p + "right.", m["right"], eps)
    return 0.5 * (unit_rms(left, eps) * W[p + "left.out"] + unit_rms(right, eps) * W[p + "right.out"])


def lightning(h, W, p, m, eps):
    """Linear attention with a fixed decay per head: S <- c_h S + k v^T, o = S^T q, silu on q, k and v; all heads normed
    together, weighted, gated and projected."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ W[p + "q"].T).view(T, H, d), silu(h @ W[p + "k"].T).view(T, H, d)
    v = silu(h @ W[p + "v"].T).view(T, H, dv)
    c = torch.tensor(m["decay"], dtype=h.dtype)[:, None, None]
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    o = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = c * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkd,hk->hd", S, q[t])
    y = unit_rms(o.reshape(T, H * dv), eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


# ---- feed-forwards ----------------------------------------------------------------------------------------
def dense_ff(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def route(h, router, top, groups, keep):
    """Chosen experts and their weights: softmax scores over all; a group counts by its best score; only the experts of
    the `keep` best groups may be chosen; the weights are the scores themselves."""
    s = torch.softmax(h @ router.T, dim=-1)
    T, E = s.shape
    size = E // groups
    best = s.view(T, groups, size).amax(-1)
    kept = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best.topk(keep, dim=-1).indices, True)
    ids = s.masked_fill(~kept.repeat_interleave(size, dim=1), -1.0).topk(top, dim=-1).indices
    return ids, s.gather(1, ids)


def expert(x, W, p):
    return (silu(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def experts_ff(h, W, p, f):
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, weights = route(h, W[p + "router"], r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        t, c = (ids == e).nonzero(as_tuple=True)
        if t.numel():
            out.index_add_(0, t, weights[t, c][:, None] * expert(h[t], W, f"{p}e{e}."))
    return out


# ---- the model ----------------------------------------------------------------------------------------------
def mix(h, W, p, layer, eps):
    if layer["type"] == "parallel":
        return side_by_side(h, W, p, layer["mixer"], eps)
    if layer["type"] == "lightning":
        return lightning(h, W, p, layer["mixer"], eps)
    raise ValueError(layer["type"])


def feed_forward(h, W, p, f):
    return dense_ff(h, W, p) if f["kind"] == "dense" else experts_ff(h, W, p, f)


def forward(cfg, weights, tokens, streams=None):
    """float64 logits [T, vocab] of a whole sequence; `streams` (a list) receives the stream after every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = offset_norm(x, W[p + "norm1"], eps)
        y = mix(input_conv(h, W[p + "canon1"]), W, p + "mix.", layer, eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(input_conv(h, W[p + "canon2"]), W, p + "mlp.", layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return offset_norm(x, W["final.norm"], eps) @ W["embed"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ---- tensors ------------------------------------------------------------------------------------------------
def tensor_shapes(cfg, ranks=None):
    """Names and shapes; `ranks` = (decay's, gate's) low rank of layer i's delta rule: a function of i (default 5 + i, 3 + 2 i)."""
    ranks = ranks or (lambda i: (5 + i, 3 + 2 * i))
    D, K = cfg["width"], cfg["canon"]["taps"]
    shapes = {"embed": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        x = p + "mix."
        shapes[p + "norm1"], shapes[p + "canon1"] = (D,), (D, K)
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            L, R = x + "left.", x + "right."
            rows = {"q": a["heads"] * a["dim"], "k": a["kv_heads"] * a["dim"], "v": a["kv_heads"] * a["vdim"]}
            for n, r in rows.items():
                shapes[L + n], shapes[L + n + ".b"], shapes[L + n + ".conv"] = (r, D), (r,), (r, a["conv"])
            shapes[L + "o"], shapes[L + "o.b"], shapes[L + "out"] = (D, a["heads"] * a["vdim"]), (D,), (D,)
            hd, hv = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            rows = {"q": b["kv_heads"] * b["dim"], "k": b["kv_heads"] * b["dim"], "v": hv}
            for n, r in rows.items():
                shapes[R + n], shapes[R + n + ".conv"] = (r, D), (r, b["conv"])
            ra, rg = ranks(i)
            shapes.update({R + "b": (b["heads"], D), R + "A_log": (b["heads"],), R + "dt_bias": (hd,), R + "a1": (ra, D),
                           R + "a2": (hd, ra), R + "g1": (rg, D), R + "g2": (hv, rg), R + "norm": (b["vdim"],),
                           R + "o": (D, hv), R + "out": (D,)})
        else:
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            shapes.update({x + "q": (H * d, D), x + "k": (H * d, D), x + "v": (H * dv, D), x + "g": (H * dv, D),
                           x + "norm": (H * dv,), x + "o": (D, H * dv)})
        if f is not None:
            shapes[p + "canon2"] = (D, K)
            if f["kind"] == "dense":
                shapes[p + "mlp.up"], shapes[p + "mlp.down"] = (f["ff"], D), (D, f["ff"])
            else:
                ff = f["expert"]["ff"]
                for e in range(f["router"]["experts"]):
                    q = f"{p}mlp.e{e}."
                    shapes[q + "gate"], shapes[q + "up"], shapes[q + "down"] = (ff, D), (ff, D), (D, ff)
                shapes[p + "mlp.router"] = (f["router"]["experts"], D)
    return shapes


def random_weights(cfg, seed, hot=1.0, ranks=None):
    """bfloat16 tensors.  Matrices N(0, hot^2 / in); offset norm weights N(0, 0.2), plain ones 1 + N(0, 0.2); short
    convolutions of unit size; decays between 0.6 and 1 per step; routers whose scores spread."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape: torch.randn(*shape, generator=g)
    out = {}
    for name, shape in tensor_shapes(cfg, ranks).items():
        last = name.rsplit(".", 1)[-1]
        if last == "norm1" or name == "final.norm":
            t = 0.2 * rn(*shape)
        elif last in ("norm", "out"):
            t = 1.0 + 0.2 * rn(*shape)
        elif last in ("canon1", "canon2"):
            t = 0.6 * rn(*shape) / math.sqrt(shape[1])
        elif last == "conv":
            t = rn(*shape) / math.sqrt(shape[1])
        elif name.endswith(".b") and len(shape) == 1:
            t = 0.3 * rn(*shape)
        elif last == "A_log":
            t = torch.log(0.5 + 1.5 * torch.rand(shape, generator=g))
        elif last == "dt_bias":
            t = -2.5 + 1.5 * torch.rand(shape, generator=g)
        elif name == "embed":
            t = rn(*shape)
        elif last == "router":
            t = rn(*shape) * (2.0 / math.sqrt(shape[-1]))
        else:
            t = rn(*shape) * (hot / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out
