"""Plain, slow restatement of the Korirax decoder LM in float64: one function per mechanism, written from the equations and
sharing no code with ``moshi_b200``.  Everything runs token by token on explicit per-request state (lists of past latents, keys
and values, the last convolution inputs, a state vector), with no tiling, batching, folding or fused step of any kind, so
agreement with the product path checks its kernels, its cache and its slot handling alike.

The design: parallel blocks ``x <- x + mixer(h) + ff(h)`` with ``h`` an RMS norm of ``x``, then a per-layer token input
``x <- x + rms(V (gelu(G x) * e)) * w`` with ``e`` the layer's part of a second embedding row of the token.  A stretch of layers may
run several times with the same weights, each pass on caches of its own and with a vector of its own added in front.  Mixers:
latent attention whose queries come through a latent too (a rotated part beside an unrotated one, one rotated key for all heads),
attention without rotation whose scores get a learned bias by distance and whose queries grow with the position, and a gated linear
recurrence of independent channels behind a short convolution.  Feed-forward: a silu-gated unit, or routed experts without a gate
(erf GELU) behind a sigmoid router with a choice correction and groups, beside a shared expert.

Notation: W width; H query heads over G key/value heads; per head q, k [dim], v [vdim].
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softmax(z):
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


# ---------------------------------------------------------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------------------------------------------------------
def rotary(dims, base, scaling=None):
    """(frequencies [dims / 2], amplitude).  scaling {factor, original, fast, slow}: frequencies that turn fewer than `slow` times
    over `original` positions are divided by factor, those that turn more than `fast` times stay, an index ramp lies between."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    if not scaling:
        return f, 1.0

    def index_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)], dtype=F64)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_adjacent(u, pos, freqs, amp):
    """u [.., 2 n]: dimension 2i turns with 2i + 1 by the angle pos * f_i, cos and sin times amp."""
    c, s = torch.cos(pos * freqs) * amp, torch.sin(pos * freqs) * amp
    out = u.clone()
    n = 2 * freqs.shape[0]
    a, b = u[..., 0:n:2], u[..., 1:n:2]
    out[..., 0:n:2] = a * c - b * s
    out[..., 1:n:2] = b * c + a * s
    return out


def distance_bucket(n, buckets, far):
    """Row of the bias table for a key n positions back: single distances in the first half, a logarithmic scale up to `far` in the
    second, the last row beyond."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (buckets - half)))


def temperature(pos, coef, every):
    """What the queries at position pos are multiplied by."""
    return 1.0 + coef * math.log(math.floor((pos + 1) / every) + 1.0)


# ---------------------------------------------------------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------------------------------------------------------
def latent_attention(p, m, h, pos, st, eps):
    H, d, rd, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    f, amp = rotary(rd, float(m["rot"]["base"]), m["rot"].get("scaling"))
    q = (p["uq"] @ rms_norm(p["dq"] @ h, p["dq.norm"], eps)).view(H, d + rd)
    qr = rotate_adjacent(q[:, d:], pos, f, amp)
    down = p["dkv"] @ h
    st.setdefault("c", []).append(rms_norm(down[:r], p["dkv.norm"], eps))
    st.setdefault("kr", []).append(rotate_adjacent(down[r:], pos, f, amp))
    C, KR = torch.stack(st["c"]), torch.stack(st["kr"])               # [n, r], [n, rd]
    K = (C @ p["uk"].T).view(-1, H, d)
    V = (C @ p["uv"].T).view(-1, H, dv)
    out = torch.stack([softmax((K[:, hh] @ q[hh, :d] + KR @ qr[hh]) * m["scale"]) @ V[:, hh] for hh in range(H)])
    return p["o"] @ (out.reshape(-1) * sigmoid(p["g"] @ h))


def attention(p, m, h, pos, st, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((p["q"] @ h + p["q.b"]).view(H, d), p["q.norm"], eps)
    if m.get("q_temp"):
        q = q * temperature(pos, float(m["q_temp"]["coef"]), m["q_temp"]["every"])
    st.setdefault("k", []).append(rms_norm((p["k"] @ h + p["k.b"]).view(G, d), p["k.norm"], eps))
    st.setdefault("v", []).append((p["v"] @ h + p["v.b"]).view(G, dv))
    K, V = torch.stack(st["k"]), torch.stack(st["v"])                 # [n, G, d], [n, G, dv]
    rows = [distance_bucket(pos - j, p["rel"].shape[0], m["bias_max"]) for j in range(pos + 1)]
    bias = p["rel"][rows]                                             # [n, H]
    out = torch.stack([softmax((K[:, hh // (H // G)] @ q[hh]) * m["scale"] + bias[:, hh]) @ V[:, hh // (H // G)] for hh in range(H)])
    return p["o"] @ (out.reshape(-1) * sigmoid(p["g"] @ h))


def causal_convolution(window, w, b):
    """window: the inputs of the last taps steps, oldest first (missing ones in front of the sequence are zero) -> sum_j w[:, j] u_j + b."""
    taps = w.shape[1]
    y = b.clone()
    for j, u in enumerate(window):
        y = y + w[:, taps - len(window) + j] * u
    return y


def block_diagonal(w, b, u):
    """w [blocks, n, n] applied to u in equal parts, plus b [blocks, n]."""
    nb, n, _ = w.shape
    return torch.cat([w[i] @ u[i * n:(i + 1) * n] + b[i] for i in range(nb)])


def rglru(p, m, h, pos, st, eps):
    y = gelu_tanh(p["y"] @ h + p["y.b"])
    taps = p["conv"].shape[1]
    st["u"] = (st.get("u", []) + [p["x"] @ h + p["x.b"]])[-taps:]
    u = causal_convolution(st["u"], p["conv"], p["conv.b"])
    r = sigmoid(block_diagonal(p["ra"], p["ra.b"], u))
    i = sigmoid(block_diagonal(p["ri"], p["ri.b"], u))
    log_a = -8.0 * r * softplus(p["lam"])
    st["S"] = torch.exp(log_a) * st.get("S", torch.zeros_like(u)) + torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    return p["o"] @ (st["S"] * y)


MIXERS = {"latent_attention": latent_attention, "attention": attention, "rglru": rglru}


# ---------------------------------------------------------------------------------------------------------------------------
# feed-forward and the per-layer token input
# ---------------------------------------------------------------------------------------------------------------------------
def silu_glu(p, h):
    g = p["gate"] @ h
    return p["down"] @ (g * sigmoid(g) * (p["up"] @ h))


def gelu_expert(up, down, h):
    return down @ gelu_erf(up @ h)


def route(z, correction, top, n_groups, keep, scale):
    """-> (chosen experts, their weights).  Scores are sigmoids; the choice adds the correction and is limited to the `keep` groups
    of neighbours whose two largest choice scores have the largest sum; the weights are the chosen plain scores over their sum."""
    s = sigmoid(z)
    choice = s + correction
    n = z.shape[0]
    per = n // n_groups
    two = [float(choice[g * per:(g + 1) * per].topk(min(2, per)).values.sum()) for g in range(n_groups)]
    best = sorted(range(n_groups), key=lambda g: -two[g])[:keep]
    allowed = [e for e in range(n) if e // per in best]
    idx = sorted(allowed, key=lambda e: -float(choice[e]))[:top]
    w = s[idx] / (s[idx].sum() + 1e-20) * scale
    return idx, w.tolist()


def experts(p, mlp, h):
    r = mlp["router"]
    gr = r.get("groups") or {}
    idx, w = route(p["router"] @ h, p["correction"], int(r["top"]), int(gr.get("count", 1)), int(gr.get("keep", 1)), float(r.get("scale", 1.0)))
    y = torch.zeros_like(h)
    for e, we in zip(idx, w):
        y = y + we * gelu_expert(p[f"e{e}.up"], p[f"e{e}.down"], h)
    if mlp.get("shared"):
        y = y + gelu_expert(p["shared.up"], p["shared.down"], h)
    return y


def token_input(p, x, e, eps):
    """What the layer adds for its token: rms(proj (gelu(gate x) * e)) * norm."""
    return rms_norm(p["proj"] @ (gelu_tanh(p["gate"] @ x) * e), p["norm"], eps)


def layer_runs(cfg):
    """[(layer, pass or None)] in the order they run; a pass number marks the first layer of a pass of the loop."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


# ---------------------------------------------------------------------------------------------------------------------------
class Oracle:
    """cfg: the dict of config.json; tensors: name -> tensor (any float type).  ``new_state()`` per request, ``step(state, token)``
    returns (logits [vocab], [x after every layer run])."""

    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.t = {k: v.detach().to("cpu", F64) for k, v in tensors.items()}
        self.eps = float(cfg["norm"]["eps"])
        self.runs = layer_runs(cfg)
        self.sub = [{s: {k[len(f"l{i}.{s}."):]: v for k, v in self.t.items() if k.startswith(f"l{i}.{s}.")} for s in ("mix", "mlp", "side")}
                    for i in range(len(cfg["layers"]))]

    def new_state(self):
        return {"pos": 0, "runs": [dict() for _ in self.runs]}

    def step(self, state, token):
        t, eps, pos = self.t, self.eps, state["pos"]
        x = t["embed"][token] * float((self.cfg.get("embedding") or {}).get("scale", 1.0))
        side = (self.cfg.get("token_side") or {}).get("dim", 0)
        trace = []
        for (i, t_pass), st in zip(self.runs, state["runs"]):
            L, p = self.cfg["layers"][i], self.sub[i]
            if t_pass is not None:
                x = x + t["loop.step"][t_pass]
            h = rms_norm(x, t[f"l{i}.norm1"], eps)
            y = MIXERS[L["type"]](p["mix"], L["mixer"], h, pos, st, eps)
            mlp = L.get("mlp")
            if mlp is not None:
                y = y + (silu_glu(p["mlp"], h) if mlp["kind"] == "dense" else experts(p["mlp"], mlp, h))
            x = x + y
            if side:
                x = x + token_input(p["side"], x, t["side.embed"][token][i * side:(i + 1) * side], eps)
            trace.append(x)
        logits = t["head"] @ rms_norm(x, t["final.norm"], eps)
        state["pos"] = pos + 1
        return logits, trace

    def run(self, tokens, state=None):
        """All tokens of one request in order -> (logits [n, vocab], layer runs [n_runs, n, W])."""
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
