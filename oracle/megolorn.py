"""Plain, slow restatement of the Megolorn decoder LM in float64: one function per mechanism, written from the equations and
sharing no code with ``moshi_b200``.  Everything runs token by token on explicit per-request state (lists of past keys and
values), with no tiling, batching or fused step of any kind, so agreement with the product path checks its kernels, its cache
and its slot handling alike.

The design: parallel blocks ``x <- x + mixer(h) + ff(h)`` with ``h`` a layer norm (weight, no bias) of ``x``.  The mixer is
differential softmax attention on positions of the query's own chunk: every head has two query / key maps over the same values,
``o = a1 - lambda a2``, normed to unit root mean square and scaled by ``1 - diff``, times a sigmoid gate per head.  A layer may
own no keys and values and read those of an earlier layer.  The feed-forward is a gated unit with bounded gate and value, or
routed experts behind a softmax router (choice correction, best groups, experts that return their input) beside a shared expert.

Notation: W width; H query heads over G key/value heads; per head and map q, k [dim]; values [vdim].
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softmax(z):
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def rotary_frequencies(dims, base, factor=1.0):
    """f_i = base^(-2i/dims) / factor."""
    return torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F64)


def rotate_adjacent(u, pos, freqs):
    """u [.., dim]: dimension 2i turns with 2i + 1 by the angle pos * f_i; dimensions from 2 * len(freqs) on pass unchanged."""
    n = freqs.shape[0]
    c, s = torch.cos(pos * freqs), torch.sin(pos * freqs)
    out = u.clone()
    a, b = u[..., 0:2 * n:2], u[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = a * c - b * s
    out[..., 1:2 * n:2] = b * c + a * s
    return out


def chunk_visible(pos, size):
    """The keys position pos sees: those of its own chunk up to itself (size None: all up to pos)."""
    return slice(0 if not size else (pos // size) * size, pos + 1)


def diff_lambda(p, diff):
    """exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number for the layer."""
    return math.exp(float((p["lq1"] * p["lk1"]).sum())) - math.exp(float((p["lq2"] * p["lk2"]).sum())) + diff


def differential_combine(a1, a2, lam, diff, eps):
    """unit-rms(a1 - lambda a2) * (1 - diff), per head."""
    return rms_unit(a1 - lam * a2, eps) * (1.0 - diff)


def project_heads(p, nm, h, heads, maps, dim):
    return (p[nm] @ h + p[nm + ".b"]).view(heads, maps, dim)


def differential_attention(p, m, h, pos, st, kv, eps):
    """st: this layer's own keys and values (filled here when the layer has projections of them); kv: the state they are read from
    (st itself, or that of the layer named by kv_from)."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {}
    f = None
    if rot.get("dims", 0):
        f = rotary_frequencies(int(rot["dims"]), float(rot["base"]), float((rot.get("scaling") or {}).get("factor", 1.0)))
    q = rms_unit(project_heads(p, "q", h, H, 2, d), eps) * p["q.norm"]
    if f is not None:
        q = rotate_adjacent(q, pos, f)
    if m.get("kv_from") is None:
        k = rms_unit(project_heads(p, "k", h, G, 2, d), eps) * p["k.norm"]
        if f is not None:
            k = rotate_adjacent(k, pos, f)
        st.setdefault("k", []).append(k)
        st.setdefault("v", []).append((p["v"] @ h + p["v.b"]).view(G, dv))
    sl = chunk_visible(pos, (m.get("mask") or {}).get("size"))
    K, V = torch.stack(kv["k"][sl]), torch.stack(kv["v"][sl])         # [n, G, 2, d], [n, G, dv]
    lam, diff = diff_lambda(p, float(m["diff"])), float(m["diff"])
    gate = sigmoid(p["g"] @ h)
    out = torch.zeros(H, dv, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        a = [softmax((K[:, g, mp] @ q[hh, mp]) * m["scale"]) @ V[:, g] for mp in (0, 1)]
        out[hh] = differential_combine(a[0], a[1], lam, diff, eps) * gate[hh]
    return p["o"] @ out.reshape(-1)


def bounded_glu(p, h, limit):
    """g = min(gate, limit), u = value clipped to +-limit: down (g sigmoid(1.702 g) (u + 1))."""
    g = torch.clamp(p["gate"] @ h, max=limit)
    u = torch.clamp(p["up"] @ h, -limit, limit)
    return p["down"] @ (g * sigmoid(1.702 * g) * (u + 1.0))


def silu_glu(p, h):
    return p["down"] @ (silu(p["gate"] @ h) * (p["up"] @ h))


def route(z, correction, top, n_groups, keep):
    """-> (chosen experts, their weights).  Scores are a softmax over everything; the choice adds the correction and is limited to
    the `keep` groups with the largest single choice score; the weights are the plain scores, not renormalised."""
    s = softmax(z)
    choice = s + correction
    n = z.shape[0]
    if n_groups > 1:
        per = n // n_groups
        best = sorted(range(n_groups), key=lambda g: -float(choice[g * per:(g + 1) * per].max()))[:keep]
        allowed = [e for e in range(n) if e // per in best]
    else:
        allowed = list(range(n))
    idx = sorted(allowed, key=lambda e: -float(choice[e]))[:top]
    return idx, [float(s[e]) for e in idx]


def experts(p, mlp, h):
    r = mlp["router"]
    E, gr = int(r["experts"]), r.get("groups") or {}
    idx, w = route(p["router"] @ h, p["correction"], int(r["top"]), int(gr.get("count", 1)), int(gr.get("keep", 1)))
    y = torch.zeros_like(h)
    for e, we in zip(idx, w):
        y = y + we * (silu_glu({k: p[f"e{e}.{k}"] for k in ("gate", "up", "down")}, h) if e < E else h)
    if mlp.get("shared") is not None:
        y = y + silu_glu({k: p[f"shared.{k}"] for k in ("gate", "up", "down")}, h)
    return y


# ---------------------------------------------------------------------------------------------------------------------------
class Oracle:
    """cfg: the dict of config.json; tensors: name -> tensor (any float type).  ``new_state()`` per request, ``step(state, token)``
    returns (logits [vocab], [x after every layer])."""

    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.t = {k: v.detach().to("cpu", F64) for k, v in tensors.items()}
        self.eps = float(cfg["norm"]["eps"])
        self.sub = [({k[len(f"l{i}.mix."):]: v for k, v in self.t.items() if k.startswith(f"l{i}.mix.")},
                     {k[len(f"l{i}.mlp."):]: v for k, v in self.t.items() if k.startswith(f"l{i}.mlp.")}) for i in range(len(cfg["layers"]))]

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.cfg["layers"]]}

    def step(self, state, token):
        t, eps, pos = self.t, self.eps, state["pos"]
        x = t["embed"][token] * float((self.cfg.get("embedding") or {}).get("scale", 1.0))
        trace = []
        for i, L in enumerate(self.cfg["layers"]):
            h = layer_norm(x, t[f"l{i}.norm1"], eps)
            src = L["mixer"].get("kv_from")
            st = state["layers"][i]
            y = differential_attention(self.sub[i][0], L["mixer"], h, pos, st, st if src is None else state["layers"][src], eps)
            mlp = L.get("mlp")
            if mlp is not None:
                y = y + (bounded_glu(self.sub[i][1], h, float(mlp["limit"])) if mlp["kind"] == "dense" else experts(self.sub[i][1], mlp, h))
            x = x + y
            trace.append(x)
        logits = t["head"] @ layer_norm(x, t["final.norm"], eps)
        state["pos"] = pos + 1
        return logits, trace

    def run(self, tokens, state=None):
        """All tokens of one request in order -> (logits [n, vocab], layers [n_layers, n, W])."""
        state = state if state is not None else self.new_state()
        lg, tr = [], []
        for tok in tokens:
            a, b = self.step(state, int(tok))
            lg.append(a)
            tr.append(torch.stack(b))
        return torch.stack(lg), torch.stack(tr, 1)

    def forward(self, tokens, return_layers=False):
        lg, tr = self.run(tokens)
        return (lg, tr) if return_layers else lg

    def greedy(self, prompt, n_new):
        """(tokens, gap between the two largest logits at every choice)."""
        st = self.new_state()
        lg, _ = self.run(prompt, st)
        out, gaps = [], []
        for _ in range(n_new):
            top = lg[-1].topk(2).values
            nxt = int(lg[-1].argmax())
            out.append(nxt)
            gaps.append(float(top[0] - top[1]))
            lg, _ = self.run([nxt], st)
        return out, gaps
