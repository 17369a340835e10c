"""Plain fp32/fp64 CPU restatement of the Vodavik design, one function per mechanism.

Test oracle only: slow, token-by-token where the mechanism is a recurrence, dense score matrices where
it is attention.  Shares no code with the product path.  Notation: ``T`` tokens, ``E`` width, ``H``
query heads, ``G`` key/value heads, ``D`` query/key size, ``U`` value size.  Every function takes and
returns tensors of one sequence; ``w`` is a dict of tensors by name, ``p`` a layer prefix such as ``l3``.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def layer_norm(x, weight, eps):
    """Centred norm with a gain and no offset; the variance divides by the number of elements."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * weight


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def query_temperature(positions, coef, every):
    """Gain of the query at each position: 1 + coef * ln(1 + floor((p + 1) / every))."""
    return torch.tensor([1.0 + coef * math.log(1 + (int(p) + 1) // every) for p in positions], dtype=torch.float64)


def linear(x, w, name, bias=False):
    y = x @ w[name].to(x.dtype).T
    return y + w[name + ".b"].to(x.dtype) if bias else y


def attention_keys_values(w, p, m, eps, h):
    """Normalised keys [T, G, D] and values [T, G, U] of a layer that owns them."""
    t = h.shape[0]
    k = linear(h, w, f"{p}.mix.k", bias=True).view(t, m["kv_heads"], m["dim"])
    v = linear(h, w, f"{p}.mix.v", bias=True).view(t, m["kv_heads"], m["vdim"])
    return rms_unit(k, eps) * w[f"{p}.mix.k.norm"].to(h.dtype), v


def attention_queries(w, p, m, eps, h, positions):
    """Normalised queries [T, H, D] with the temperature of their positions."""
    q = linear(h, w, f"{p}.mix.q", bias=True).view(h.shape[0], m["heads"], m["dim"])
    q = rms_unit(q, eps) * w[f"{p}.mix.q.norm"].to(h.dtype)
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(positions, temp["coef"], temp["every"]).to(h.dtype)[:, None, None]
    return q


def sink_softmax(scores, sink):
    """Softmax over the last axis whose denominator also holds exp(sink): scores [H, T, S], sink [H]."""
    s = sink.to(scores.dtype)[:, None, None]
    top = torch.maximum(scores.amax(-1, keepdim=True), s)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(s - top))


def causal_sink_attention(q, k, v, scale, sink, first_pos):
    """q [T, H, D] at positions first_pos..., k [S, G, D], v [S, G, U] from position 0 -> [T, H, U]."""
    t, heads, _ = q.shape
    rep = heads // k.shape[1]
    kk, vv = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    scores = torch.einsum("thd,shd->hts", q, kk) * scale
    later = torch.arange(k.shape[0])[None, :] > (first_pos + torch.arange(t))[:, None]
    probs = sink_softmax(scores.masked_fill(later[None], -math.inf), sink)
    return torch.einsum("hts,shu->thu", probs, vv)


def attention_mixer(w, p, m, eps, h, first_pos, cache):
    """``cache`` maps layer prefixes to their (keys, values) so far; a layer with ``kv_from`` reads
    another layer's entry."""
    t = h.shape[0]
    if m.get("kv_from") is None:
        k, v = attention_keys_values(w, p, m, eps, h)
        if p in cache:
            k, v = torch.cat([cache[p][0], k]), torch.cat([cache[p][1], v])
        cache[p] = (k, v)
        src = p
    else:
        src = f"l{m['kv_from']}"
    k, v = cache[src]
    q = attention_queries(w, p, m, eps, h, range(first_pos, first_pos + t))
    o = causal_sink_attention(q, k, v, m["scale"], w[f"{p}.mix.sink"], first_pos).reshape(t, -1)
    return linear(o * torch.sigmoid(linear(h, w, f"{p}.mix.g")), w, f"{p}.mix.o")


def mlstm_gates(w, p, cap, h):
    """Log input gate and log forget gate, [T, H] each."""
    i = cap * torch.tanh(linear(h, w, f"{p}.mix.i", bias=True) / cap)
    f = F.logsigmoid(cap * torch.tanh(linear(h, w, f"{p}.mix.f", bias=True) / cap))
    return i, f


def mlstm_recurrence(q, k, v, i, f, state):
    """q, k [T, H, D], v [T, H, U], gates [T, H]; ``state`` = (S [H, D, U], n [H, D], m [H]) or None.
    Returns outputs [T, H, U] before the head norm, and the new state."""
    t, heads, dim = q.shape
    if state is None:
        state = (q.new_zeros(heads, dim, v.shape[-1]), q.new_zeros(heads, dim), q.new_zeros(heads))
    s, n, m = state
    out = []
    for a in range(t):
        m_new = torch.maximum(f[a] + m, i[a])
        keep, add = torch.exp(f[a] + m - m_new), torch.exp(i[a] - m_new)
        s = keep[:, None, None] * s + add[:, None, None] * k[a][:, :, None] * v[a][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[a]
        m = m_new
        num = torch.einsum("hdu,hd->hu", s, q[a])
        den = torch.maximum((n * q[a]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(num / den[:, None])
    return torch.stack(out), (s, n, m)


def mlstm_mixer(w, p, m, eps, h, states):
    t, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w, f"{p}.mix.q").view(t, heads, dim) * dim ** -0.5
    k = linear(h, w, f"{p}.mix.k").view(t, heads, dim)
    v = linear(h, w, f"{p}.mix.v").view(t, heads, vdim)
    i, f = mlstm_gates(w, p, m["gate_cap"], h)
    o, states[p] = mlstm_recurrence(q, k, v, i, f, states.get(p))
    o = rms_unit(o, eps).reshape(t, -1) * w[f"{p}.mix.norm"].to(h.dtype)
    return linear(o * torch.sigmoid(linear(h, w, f"{p}.mix.g")), w, f"{p}.mix.o")


def feed_forward(w, p, h):
    return linear(F.relu(linear(h, w, f"{p}.mlp.up")) ** 2, w, f"{p}.mlp.down")


class Sequence:
    """One sequence's caches; ``step`` feeds its next tokens and returns their logits [T, vocab]."""

    def __init__(self, config: dict, weights: dict, dtype=torch.float32):
        self.c, self.w, self.dtype = config, weights, dtype
        self.pos, self.cache, self.states = 0, {}, {}
        self.residuals: list[torch.Tensor] = []     # after every layer, of the last step

    def step(self, tokens) -> torch.Tensor:
        c, w = self.c, self.w
        eps, alpha = c["norm"]["eps"], c["postln_alpha"]
        x = w["embed"].to(self.dtype)[torch.as_tensor(tokens, dtype=torch.long)]
        self.residuals = []
        for n, layer in enumerate(c["layers"]):
            p = f"l{n}"
            if layer["type"] == "attention":
                y = attention_mixer(w, p, layer["mixer"], eps, x, self.pos, self.cache)
            else:
                y = mlstm_mixer(w, p, layer["mixer"], eps, x, self.states)
            x = layer_norm(alpha * x + y, w[f"{p}.norm1"].to(self.dtype), eps)
            if layer["mlp"] is not None:
                x = layer_norm(alpha * x + feed_forward(w, p, x), w[f"{p}.norm2"].to(self.dtype), eps)
            self.residuals.append(x)
        self.pos += len(tokens)
        x = layer_norm(x, w["final.norm"].to(self.dtype), eps)
        return linear(x, w, "head") * c["logit_scale"]


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

    mat("embed", config["vocab"], width, 1.0)
    for n, layer in enumerate(config["layers"]):
        p, m = f"l{n}", layer["mixer"]
        h, d, u = m["heads"], m["dim"], m["vdim"]
        vec(f"{p}.norm1", width, 1.0)
        if layer["type"] == "attention":
            mat(f"{p}.mix.q", h * d, width)
            vec(f"{p}.mix.q.b", h * d)
            vec(f"{p}.mix.q.norm", d, 1.2, 0.3)
            if m.get("kv_from") is None:
                kv = m["kv_heads"]
                mat(f"{p}.mix.k", kv * d, width)
                vec(f"{p}.mix.k.b", kv * d)
                vec(f"{p}.mix.k.norm", d, 1.2, 0.3)
                mat(f"{p}.mix.v", kv * u, width)
                vec(f"{p}.mix.v.b", kv * u)
            vec(f"{p}.mix.sink", h, 2.0, 1.0)
        else:
            mat(f"{p}.mix.q", h * d, width)
            mat(f"{p}.mix.k", h * d, width)
            mat(f"{p}.mix.v", h * u, width)
            mat(f"{p}.mix.i", h, width)
            vec(f"{p}.mix.i.b", h, 0.0, 1.0)
            mat(f"{p}.mix.f", h, width)
            vec(f"{p}.mix.f.b", h, 3.5, 2.0)
            vec(f"{p}.mix.norm", h * u, 1.0)
        mat(f"{p}.mix.g", h * u, width)
        mat(f"{p}.mix.o", width, h * u)
        if layer["mlp"] is not None:
            vec(f"{p}.norm2", width, 1.0)
            mat(f"{p}.mlp.up", layer["mlp"]["ff"], width)
            mat(f"{p}.mlp.down", width, layer["mlp"]["ff"])
    vec("final.norm", width, 1.0)
    mat("head", config["vocab"], width)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
