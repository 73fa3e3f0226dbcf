"""The Pagulix decoder restated plainly: float64 torch on the CPU, whole sequences at once, one function per mechanism,
no cache, no batching, no code shared with the library.  The tests compare the engine with this.

Notation: T tokens, D the stream's width, S parallel streams; W["name"] the tensors under the names of the weight file
(matrices [out, in]); t is a query's position and s a key's, both counted from 0.
"""
import math

import torch


# ---- small pieces ---------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def short_conv(u, taps):
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), nothing before the sequence's start."""
    T = u.shape[0]
    K = taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(K):
        back = K - 1 - j
        if back < T:
            y[back:] += taps[:, j] * u[:T - back]
    return y


# ---- rotation -------------------------------------------------------------------------------------------
def frequencies(dims, base):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)


def stretched(f, scaling):
    """Long waves are slowed by `factor`, short ones kept, and between the two bounds both are blended by how often a
    wave turns over the original context."""
    out = []
    for x in f.tolist():
        wave = 2.0 * math.pi / x
        turns = scaling["original"] / wave
        if turns > scaling["high"]:
            out.append(x)
        elif turns < scaling["low"]:
            out.append(x / scaling["factor"])
        else:
            s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1.0 - s) * x / scaling["factor"] + s * x)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, f, interleaved):
    """x [T, heads, dim]: the first 2 len(f) channels turned by (position * f), the rest unchanged."""
    T, n = x.shape[0], len(f)
    angle = torch.arange(T, dtype=torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    y = x.clone()
    if interleaved:
        u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
        y[..., 0:2 * n:2], y[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :n], x[..., n:2 * n]
        y[..., :n], y[..., n:2 * n] = u * c - v * s, v * c + u * s
    return y


# ---- mixers ---------------------------------------------------------------------------------------------
def masked_softmax(scores, visible, sink=None):
    """scores [H, T, T]; `sink` [H]: one more term exp(sink_h) of the denominator."""
    scores = scores.masked_fill(~visible[None], float("-inf"))
    top = scores.amax(-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


def distances(T):
    t = torch.arange(T)
    return t[:, None] - t[None, :]


def latent_attention(h, W, p, m, eps):
    """Keys and values of every head from one latent row per position; part of the key is rotated and shared; a window and
    a sink per head."""
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    f = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q = (h @ W[p + "q"].T).view(T, H, d + r)
    q_plain, q_rot = q[..., :d], rotate(q[..., d:], f, interleaved=True)
    down = h @ W[p + "dkv"].T
    c = rms_norm(down[:, :rank], W[p + "dkv.norm"], eps)
    k_rot = rotate(down[:, None, rank:], f, interleaved=True)[:, 0]
    k_plain = (c @ W[p + "uk"].T).view(T, H, d)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    scores = (torch.einsum("thd,shd->hts", q_plain, k_plain) + torch.einsum("thd,sd->hts", q_rot, k_rot)) * m["scale"]
    back = distances(T)
    visible = back >= 0
    if m.get("mask") is not None:
        visible = visible & (back < m["mask"]["size"])
    w = masked_softmax(scores, visible, W[p + "sink"])
    return torch.einsum("hts,shd->thd", w, v).reshape(T, H * dv) @ W[p + "o"].T


def mixed_values(v, lam, first):
    return (1.0 - lam) * v + lam * first


def attention(h, W, p, m, eps, shared):
    """Grouped heads; q and k are made unit-RMS after the rotation; values blended with those of the first mixing layer
    (kept in `shared`)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"]["dims"], m["rot"]["base"])
    if m["rot"].get("scaling") is not None:
        f = stretched(f, m["rot"]["scaling"])
    q = unit_rms(rotate((h @ W[p + "q"].T).view(T, H, d), f, interleaved=False), eps)
    k = unit_rms(rotate((h @ W[p + "k"].T).view(T, G, d), f, interleaved=False), eps)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    if m.get("v_mix"):
        if "values" in shared:
            v = mixed_values(v, W[p + "vmix"], shared["values"])
        else:
            shared["values"] = v
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    w = masked_softmax(torch.einsum("thd,shd->hts", q, k) * m["scale"], distances(T) >= 0)
    return torch.einsum("hts,shd->thd", w, v).reshape(T, H * dv) @ W[p + "o"].T


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(h, W, p, m, eps):
    """Per head a state S [d, dv];  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vectors(q.view(T, G, d)) * d ** -0.5
    k = unit_vectors(k.view(T, G, d))
    q, k, v = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1), v.view(T, H, dv)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    o = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkd,hk->hd", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkd,hk->hd", S, q[t])
    gate = silu(h @ W[p + "g"].T).view(T, H, dv)
    return (rms_norm(o, W[p + "norm"], eps) * gate).reshape(T, H * dv) @ W[p + "o"].T


def mix(h, W, p, layer, eps, shared):
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return latent_attention(h, W, p, m, eps)
    if layer["type"] == "attention":
        return attention(h, W, p, m, eps, shared)
    if layer["type"] == "delta":
        return delta_rule(h, W, p, m, eps)
    raise ValueError(layer["type"])


# ---- feed-forward -----------------------------------------------------------------------------------------
def route(h, router, bias, top):
    """The `top` largest biased logits and the softmax over just them."""
    z = h @ router.T + bias
    chosen = z.topk(top, dim=-1)
    return chosen.indices, torch.softmax(chosen.values, dim=-1)


def expert(x, W, p):
    return (silu(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def feed_forward(h, W, p, f):
    ids, weights = route(h, W[p + "router"], W[p + "router.b"], f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, c = (ids == e).nonzero(as_tuple=True)
        if t.numel():
            out.index_add_(0, t, weights[t, c][:, None] * expert(h[t], W, f"{p}e{e}."))
    if f.get("shared") is not None:
        out = out + expert(h, W, p + "shared.")
    return out


# ---- streams ----------------------------------------------------------------------------------------------
def read_streams(x, w):
    """x [S, T, D], w [S]: the sublayer's input."""
    return torch.einsum("s,std->td", w, x)


def write_streams(x, mixing, out, y, factor):
    """mixing [from, to]: every stream becomes a sum of all old ones and its share of the sublayer's result."""
    return torch.einsum("st,snd->tnd", mixing, x) + factor * out[:, None, None] * y[None]


# ---- the model ----------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, streams=None):
    """float64 logits [T, vocab] of a whole sequence; `streams` (a list) receives the sum of the streams after every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps, factor = cfg["norm"]["eps"], cfg["residual_mult"]
    e = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = e[None].repeat(cfg["streams"], 1, 1)
    shared = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        u = read_streams(x, W[p + "hc1.in"])
        y = mix(rms_norm(u, W[p + "norm1"], eps), W, p + "mix.", layer, eps, shared) * W[p + "ls1"]
        x = write_streams(x, W[p + "hc1.mix"], W[p + "hc1.out"], y, factor)
        if layer.get("mlp") is not None:
            u = read_streams(x, W[p + "hc2.in"])
            y = feed_forward(rms_norm(u, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"]) * W[p + "ls2"]
            x = write_streams(x, W[p + "hc2.mix"], W[p + "hc2.out"], y, factor)
        if streams is not None:
            streams.append(x.sum(0))
    z = rms_norm(x.sum(0), W["final.norm"], eps) @ W["embed"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)


def greedy(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ---- tensors ------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    D, S = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        x = p + "mix."

        def around(q):
            shapes.update({f"{p}norm{q}": (D,), f"{p}ls{q}": (D,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,),
                           f"{p}hc{q}.mix": (S, S)})
        around(1)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            r, rank = m["rot_dim"], m["kv_rank"]
            shapes.update({x + "q": (H * (d + r), D), x + "dkv": (rank + r, D), x + "dkv.norm": (rank,), x + "uk": (H * d, rank),
                           x + "uv": (H * dv, rank), x + "sink": (H,), x + "o": (D, H * dv)})
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            shapes.update({x + "q": (H * d, D), x + "k": (G * d, D), x + "v": (G * dv, D), x + "o": (D, H * dv)})
            if m.get("v_mix"):
                shapes[x + "vmix"] = ()
        else:
            G = m["kv_heads"]
            for n, rows in {"q": G * d, "k": G * d, "v": H * dv}.items():
                shapes[x + n], shapes[x + n + ".conv"] = (rows, D), (rows, m["conv"])
            shapes.update({x + "b": (H, D), x + "a": (H, D), x + "A_log": (H,), x + "dt_bias": (H,), x + "g": (H * dv, D),
                           x + "norm": (dv,), x + "o": (D, H * dv)})
        if f is not None:
            around(2)
            q = p + "mlp."
            experts = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
            if f.get("shared") is not None:
                experts["shared."] = f["shared"]["ff"]
            for name, ff in experts.items():
                shapes[q + name + "gate"], shapes[q + name + "up"], shapes[q + name + "down"] = (ff, D), (ff, D), (D, ff)
            shapes[q + "router"], shapes[q + "router.b"] = (f["router"]["experts"], D), (f["router"]["experts"],)
    return shapes


def random_weights(cfg, seed, hot=1.0):
    """bfloat16 tensors.  Matrices N(0, hot^2 / in); norm weights and layer scales 1 + N(0, 0.2); stream readings, writings and
    mixings that differ between streams; decays between 0.6 and 1 per step; routers whose logits spread."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape: torch.randn(*shape, generator=g)
    S = cfg["streams"]
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm", "ls1", "ls2"):
            t = 1.0 + 0.2 * rn(*shape)
        elif last == "in":
            t = (1.0 + 0.5 * rn(*shape)) / S
        elif last == "out":
            t = 1.0 + 0.5 * rn(*shape)
        elif ".hc" in name and last == "mix":
            t = torch.eye(S) + 0.2 * rn(*shape) / math.sqrt(S)
        elif last == "conv":
            t = rn(*shape) / math.sqrt(shape[1])
        elif last == "b" and len(shape) == 1:
            t = 0.5 * rn(*shape)
        elif last == "vmix":
            t = 0.2 + 0.6 * torch.rand((), generator=g)
        elif last == "sink":
            t = rn(*shape)
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
