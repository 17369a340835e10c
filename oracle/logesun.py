"""Plain CPU restatement of the Logesun design, one function per mechanism.

Test oracle only: dense score matrices, one expert after the other, every key and value spelled out per head.
Shares no code with the product path.  Notation: ``T`` tokens, ``S`` cached positions, ``E`` width, ``H`` heads,
``D`` unrotated and ``R`` rotated query/key size, ``U`` value size, ``C`` latent size.  Every function takes and
returns tensors of one sequence; ``w`` is a dict of tensors by name, ``p`` a layer prefix such as ``l3``.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight.to(x.dtype)


def linear(x, w, name):
    return x @ w[name].to(x.dtype).T


def rotate_pairs(x, positions, base, dims):
    """Rotates neighbours (2i, 2i + 1) of the first ``dims`` of the last axis by position * base^(-2i / dims).
    x [T, ..., R] with one position per row."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    angle = torch.as_tensor(positions, dtype=torch.float64)[:, None] * base ** (-2.0 * i / dims)
    angle = angle.reshape(len(angle), *[1] * (x.dim() - 2), dims // 2)
    c, s = torch.cos(angle).to(x.dtype), torch.sin(angle).to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def window_mask(first_pos, n_queries, n_keys, size):
    """True where query row t (position first_pos + t) may see key s: 0 <= distance < size."""
    d = (first_pos + torch.arange(n_queries))[:, None] - torch.arange(n_keys)[None, :]
    return (d >= 0) & (d < size)


def sink_softmax(scores, sink):
    """Softmax over the last axis whose denominator also holds exp(sink): scores [H, T, S], sink [H]."""
    s = sink.to(scores.dtype)[:, None, None]
    top = torch.maximum(scores.amax(-1, keepdim=True), s)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(s - top))


def latent_queries(w, p, m, eps, h, positions):
    """Unrotated [T, H, D] and rotated [T, H, R] parts of the queries."""
    q = linear(rms_norm(linear(h, w, f"{p}.mix.dq"), w[f"{p}.mix.dq.norm"], eps), w, f"{p}.mix.uq")
    q = q.view(h.shape[0], m["heads"], m["dim"] + m["rot_dim"])
    return q[..., :m["dim"]], rotate_pairs(q[..., m["dim"]:], positions, m["rot"]["base"], m["rot"]["dims"])


def latent_rows(w, p, m, eps, h, positions):
    """What is cached of every token: the normed latent [T, C] and the rotated key part [T, R]."""
    y = linear(h, w, f"{p}.mix.dkv")
    c = rms_norm(y[:, :m["kv_rank"]], w[f"{p}.mix.dkv.norm"], eps)
    return c, rotate_pairs(y[:, m["kv_rank"]:], positions, m["rot"]["base"], m["rot"]["dims"])


def latent_attention(w, p, m, eps, h, first_pos, cache, key):
    t, heads = h.shape[0], m["heads"]
    positions = range(first_pos, first_pos + t)
    c, kr = latent_rows(w, p, m, eps, h, positions)
    if key in cache:
        c, kr = torch.cat([cache[key][0], c]), torch.cat([cache[key][1], kr])
    cache[key] = (c, kr)
    qn, qr = latent_queries(w, p, m, eps, h, positions)
    k = linear(c, w, f"{p}.mix.uk").view(-1, heads, m["dim"])
    v = linear(c, w, f"{p}.mix.uv").view(-1, heads, m["vdim"])
    scores = (torch.einsum("thd,shd->hts", qn, k) + torch.einsum("thr,sr->hts", qr, kr)) * m["scale"]
    seen = window_mask(first_pos, t, c.shape[0], m["mask"]["size"])
    probs = sink_softmax(scores.masked_fill(~seen[None], -math.inf), w[f"{p}.mix.sink"])
    return linear(torch.einsum("hts,shu->thu", probs, v).reshape(t, -1), w, f"{p}.mix.o")


def gated_silu(w, p, h):
    g = linear(h, w, f"{p}.gate")
    return linear(g * torch.sigmoid(g) * linear(h, w, f"{p}.up"), w, f"{p}.down")


def clamped_expert(w, p, limit, h):
    g = linear(h, w, f"{p}.gate").clamp(max=limit)
    u = linear(h, w, f"{p}.up").clamp(-limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), w, f"{p}.down")


def route(w, p, top, h):
    """Chosen experts [T, top] (largest score first) and their scores, which are the weights."""
    scores = torch.sigmoid(linear(h, w, f"{p}.mlp.router"))
    weight, chosen = scores.topk(top, -1)
    return chosen, weight


def mixture(w, p, m, h):
    chosen, weight = route(w, p, m["router"]["top"], h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t].tolist(), weight[t]):
            out[t] += clamped_expert(w, f"{p}.mlp.e{e}", m["expert"]["limit"], a * h[t:t + 1])[0]
    if m.get("shared") is not None:
        out = out + clamped_expert(w, f"{p}.mlp.shared", m["shared"]["limit"], h)
    return out


def layer_runs(config):
    """(layer, pass, embedding added ahead of it) in the order in which layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return [(i, 0, False) for i in range(n)]
    lo, hi = loop["start"], loop["stop"]
    runs = [(i, 0, False) for i in range(lo)]
    for k in range(loop["times"]):
        runs += [(i, k, k > 0 and i == lo) for i in range(lo, hi)]
    return runs + [(i, 0, False) for i in range(hi, n)]


class Sequence:
    """One sequence's caches; ``step`` feeds its next tokens and returns their logits [T, vocab]."""

    def __init__(self, config: dict, weights: dict, dtype=torch.float32):
        self.c, self.w, self.dtype = config, weights, dtype
        self.pos, self.cache = 0, {}
        self.residuals: list[torch.Tensor] = []     # after every layer run, of the last step

    def step(self, tokens) -> torch.Tensor:
        c, w = self.c, self.w
        eps = c["norm"]["eps"]
        emb = w["embed"].to(self.dtype)[torch.as_tensor(tokens, dtype=torch.long)]
        x = emb
        self.residuals = []
        for n, turn, add in layer_runs(c):
            p, layer = f"l{n}", c["layers"][n]
            if add:
                x = x + emb
            y = latent_attention(w, p, layer["mixer"], eps, rms_norm(x, w[f"{p}.norm1"], eps), self.pos, self.cache, (n, turn))
            x = x + rms_norm(y, w[f"{p}.norm1b"], eps)
            m = layer["mlp"]
            if m is not None:
                h = rms_norm(x, w[f"{p}.norm2"], eps)
                y = gated_silu(w, f"{p}.mlp", h) if m["kind"] == "dense" else mixture(w, p, m, h)
                x = x + rms_norm(y, w[f"{p}.norm2b"], eps)
            self.residuals.append(x)
        self.pos += len(tokens)
        return linear(rms_norm(x, w["final.norm"], eps), w, "head")


def greedy(config, weights, prompt, n_new, dtype=torch.float32):
    """Greedy continuation: (tokens, logits of the step that chose each token)."""
    seq = Sequence(config, weights, dtype)
    logits = seq.step(prompt)[-1]
    toks, rows = [], []
    for _ in range(n_new):
        rows.append(logits)
        toks.append(int(logits.argmax()))
        logits = seq.step([toks[-1]])[-1]
    return toks, torch.stack(rows)


def random_weights(config, seed, gain=1.0):
    """Seeded bf16-rounded weights by tensor name for a configuration."""
    g = torch.Generator().manual_seed(seed)
    width = config["width"]
    w = {}

    def mat(name, rows, cols, std=None):
        w[name] = torch.randn(rows, cols, generator=g) * (std if std is not None else gain / math.sqrt(cols))

    def vec(name, n, mean=0.0, std=0.2):
        w[name] = mean + std * torch.randn(n, generator=g)

    def ffn(name, ff):
        mat(f"{name}.gate", ff, width)
        mat(f"{name}.up", ff, width)
        mat(f"{name}.down", width, ff)

    mat("embed", config["vocab"], width, 1.0)
    for n, layer in enumerate(config["layers"]):
        p, m, f = f"l{n}", layer["mixer"], layer["mlp"]
        h = m["heads"]
        vec(f"{p}.norm1", width, 1.0)
        vec(f"{p}.norm1b", width, 0.7)
        mat(f"{p}.mix.dq", m["q_rank"], width)
        vec(f"{p}.mix.dq.norm", m["q_rank"], 1.5, 0.3)
        mat(f"{p}.mix.uq", h * (m["dim"] + m["rot_dim"]), m["q_rank"])
        mat(f"{p}.mix.dkv", m["kv_rank"] + m["rot_dim"], width)
        vec(f"{p}.mix.dkv.norm", m["kv_rank"], 1.5, 0.3)
        mat(f"{p}.mix.uk", h * m["dim"], m["kv_rank"])
        mat(f"{p}.mix.uv", h * m["vdim"], m["kv_rank"])
        vec(f"{p}.mix.sink", h, 2.0, 1.0)
        mat(f"{p}.mix.o", width, h * m["vdim"])
        if f is None:
            continue
        vec(f"{p}.norm2", width, 1.0)
        vec(f"{p}.norm2b", width, 0.7)
        if f["kind"] == "dense":
            ffn(f"{p}.mlp", f["ff"])
        else:
            mat(f"{p}.mlp.router", f["router"]["experts"], width)
            for e in range(f["router"]["experts"]):
                ffn(f"{p}.mlp.e{e}", f["expert"]["ff"])
            if f.get("shared") is not None:
                ffn(f"{p}.mlp.shared", f["shared"]["ff"])
    vec("final.norm", width, 1.0)
    mat("head", config["vocab"], width)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
