"""Plain, slow restatement of the Tolanex decoder, one function per mechanism, for the tests.

Tolanex is a decoder-only model given as a list of layers.  The stream starts as the sum of three table rows: the
token's, the bigram's and the position's.  The bigram row of (previous token p, token c) is
(p * mul_prev + c * mul_cur) mod buckets; a sequence's first token has no predecessor and takes row `buckets`, the last one.
Sublayers read the stream itself; only their OUTPUT is normed:

    x <- x + m * (rms(mixer(x)) * w1);   x <- x + m * (rms(ff(x)) * w2)      (the second line only when the layer has a feed-forward)

with one constant m for the model.  The logits are head . (rms(x) * w_final).

Mixers:

* "delta": the gated delta rule with ONE decay per head.  q, k (kv_heads x dim) and v (heads x vdim) each pass a short causal
  convolution over time and silu; q and k heads become unit vectors (x / sqrt(sum x^2 + 1e-6)), q is scaled by dim^(-1/2).
  beta = sigmoid(B x), g = exp(-exp(A_log) softplus(A x + dt_bias)), one number per head each.  Per head, S [dim, vdim] from zero:
      S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
  o is divided by its root mean square per head, multiplied by a gain shared by the heads and by silu(G x), and projected.
* "latent_attention": q = W_q x per head; a latent c = rms(W_dkv x) * gain per token (the only thing a cache needs); k = U_k c and
  v = U_v c per head; no positions in the scores; (q . k) * scale; causal softmax; projected.  A layer with "kv_from": j has no W_dkv
  and attends over the latents layer j produced, with queries and up-projections of its own.

Feed-forward "moe": scores softmax(R x) over all experts; experts form equal groups of neighbours, a group scores its largest score and
only the best `keep` groups may supply experts; of those the `top` with the largest scores are used, each weighted by its score times
router.scale (not renormalised).  An expert is W_down (silu(W_gate x) * (W_up x)).  A shared expert of the same form, multiplied by
sigmoid(W_sg x), is added.

Nothing here shares code with the engine.  Tensors go in as a dict of torch tensors under the checkpoint's names.
`Stepper` runs token by token from explicit state (cached latents, matrix states, the last inputs of the convolutions, the
previous token); `forward` feeds a whole sequence through it.
"""
from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6          # q and k of the delta rule: x / sqrt(sum(x^2) + UNIT_EPS)


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def bigram_row(prev: int | None, cur: int, buckets: int, mul_prev: int, mul_cur: int) -> int:
    """Row of the bigram table; prev None = the first token of a sequence."""
    return buckets if prev is None else (prev * mul_prev + cur * mul_cur) % buckets


def embed(w: dict, emb: dict, prev: int | None, cur: int, pos: int) -> torch.Tensor:
    bg = emb["bigram"]
    return w["embed"][cur] + w["bigram"][bigram_row(prev, cur, bg["buckets"], bg["mul_prev"], bg["mul_cur"])] + w["pos"][pos]


def out_norm_add(x: torch.Tensor, y: torch.Tensor, gain: torch.Tensor, m: float, eps: float) -> torch.Tensor:
    return x + m * rms_norm(y, gain, eps)


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def conv_step(hist: torch.Tensor, x: torch.Tensor, taps_w: torch.Tensor):
    """hist [taps - 1, C] the inputs before x [C] (oldest first); taps_w [C, taps], last column for x.  -> (new hist, output [C])."""
    ext = torch.cat([hist, x[None]], 0)
    return ext[1:], (taps_w.T * ext).sum(0)


def head_decay(a: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor) -> torch.Tensor:
    return torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(a + dt_bias))


def delta_step(S, q, k, v, g, beta):
    """One head: S [dim, vdim], g and beta numbers.  -> (S', o [vdim])."""
    S = g * S
    u = beta * (v - S.T @ k)
    S = S + k[:, None] * u[None, :]
    return S, S.T @ q


def latent_attention_step(q, lat, uk, uv, heads, dim, vdim, scale):
    """The newest query q [heads*dim] over latents lat [n, rank] (its own is the last).  Keys and values are rebuilt per head."""
    keys, values = lat @ uk.T, lat @ uv.T
    out = []
    for a in range(heads):
        s = (keys[:, a * dim:(a + 1) * dim] @ q[a * dim:(a + 1) * dim]) * scale
        out.append(torch.softmax(s, 0) @ values[:, a * vdim:(a + 1) * vdim])
    return torch.cat(out)


def gated_expert(x: torch.Tensor, w: dict, pre: str) -> torch.Tensor:
    return w[pre + "down"] @ (silu(w[pre + "gate"] @ x) * (w[pre + "up"] @ x))


def route(z: torch.Tensor, top: int, count: int, keep: int, scale: float):
    """Router logits z [experts] -> (expert indices, weights), lowest index first on ties."""
    s = torch.softmax(z, 0)
    n = s.numel()
    per = n // count
    gs = [max(float(v) for v in s[g * per:(g + 1) * per]) for g in range(count)]
    kept = set(sorted(range(count), key=lambda g: (-gs[g], g))[:keep])
    order = sorted((e for e in range(n) if e // per in kept), key=lambda e: (-float(s[e]), e))[:top]
    return order, [s[e] * scale for e in order]


def moe_ff(x: torch.Tensor, w: dict, pre: str, mlp: dict) -> torch.Tensor:
    """x [W]."""
    ro = mlp["router"]
    gr = ro.get("groups") or {"count": 1, "keep": 1}
    idx, wt = route(w[pre + "router"] @ x, ro["top"], gr["count"], gr["keep"], ro.get("scale", 1.0))
    out = torch.zeros_like(x)
    for e, s in zip(idx, wt):
        out = out + s * gated_expert(x, w, "%se%d." % (pre, e))
    if mlp.get("shared"):
        out = out + torch.sigmoid(w[pre + "shared.sg"] @ x) * gated_expert(x, w, pre + "shared.")
    return out


class Stepper:
    """Token-by-token evaluation from explicit state."""

    def __init__(self, cfg: dict, w: dict, dtype=torch.float64):
        self.cfg = cfg
        self.w = {k: v.to(dtype) for k, v in w.items()}
        self.dtype = dtype
        self.state = [dict() for _ in cfg["layers"]]
        self.prev, self.pos = None, 0
        self.trace = []          # residual stream after every layer of the last token

    def delta(self, st, x, m, pre, eps):
        w = self.w
        H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
        parts = {}
        for n in ("q", "k", "v"):
            cw = w[pre + n + ".conv"]
            hist = st.get(n, torch.zeros(cw.shape[1] - 1, cw.shape[0], dtype=self.dtype))
            st[n], y = conv_step(hist, w[pre + n] @ x, cw)
            parts[n] = silu(y)
        q = unit_vector(parts["q"].reshape(G, D)) * D ** -0.5
        k = unit_vector(parts["k"].reshape(G, D))
        v = parts["v"].reshape(H, V)
        beta = torch.sigmoid(w[pre + "b"] @ x)
        g = head_decay(w[pre + "a"] @ x, w[pre + "A_log"], w[pre + "dt_bias"])
        gate = silu(w[pre + "g"] @ x).reshape(H, V)
        if "S" not in st:
            st["S"] = [torch.zeros(D, V, dtype=self.dtype) for _ in range(H)]
        outs = []
        for a in range(H):
            c = a // (H // G)
            st["S"][a], o = delta_step(st["S"][a], q[c], k[c], v[a], g[a], beta[a])
            outs.append(rms_norm(o, w[pre + "norm"], eps) * gate[a])
        return w[pre + "o"] @ torch.cat(outs)

    def latent(self, li, x, m, pre, eps):
        w, src = self.w, m.get("kv_from")
        if src is None:
            st = self.state[li]
            c = rms_norm(w[pre + "dkv"] @ x, w[pre + "dkv.norm"], eps)
            st["c"] = c[None] if "c" not in st else torch.cat([st["c"], c[None]], 0)
            lat = st["c"]
        else:
            lat = self.state[src]["c"]
        o = latent_attention_step(w[pre + "q"] @ x, lat, w[pre + "uk"], w[pre + "uv"], m["heads"], m["dim"], m["vdim"], m["scale"])
        return w[pre + "o"] @ o

    def step(self, token: int) -> torch.Tensor:
        """Appends one token; returns its logits."""
        cfg, w = self.cfg, self.w
        eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
        x = embed(w, cfg["embedding"], self.prev, token, self.pos)
        self.prev, self.pos = token, self.pos + 1
        self.trace = []
        for i, L in enumerate(cfg["layers"]):
            pre = "l%d." % i
            if L["type"] == "delta":
                y = self.delta(self.state[i], x, L["mixer"], pre + "mix.", eps)
            elif L["type"] == "latent_attention":
                y = self.latent(i, x, L["mixer"], pre + "mix.", eps)
            else:
                raise ValueError("mixer type %r" % L["type"])
            x = out_norm_add(x, y, w[pre + "norm1"], mult, eps)
            if L.get("mlp"):
                x = out_norm_add(x, moe_ff(x, w, pre + "mlp.", L["mlp"]), w[pre + "norm2"], mult, eps)
            self.trace.append(x)
        return w["head"] @ rms_norm(x, w["final.norm"], eps)

    def greedy(self, prompt, n: int):
        """Feeds the prompt, then n times the most likely token (lowest index on ties); returns the n tokens."""
        for t in prompt:
            y = self.step(int(t))
        out = []
        for _ in range(n):
            out.append(int(torch.argmax(y)))
            y = self.step(out[-1])
        return out


def forward(cfg: dict, w: dict, tokens, dtype=torch.float64):
    """-> (logits [T, vocab], residual stream after every layer [layers, T, W])."""
    s = Stepper(cfg, w, dtype)
    logits, traces = [], []
    for t in tokens:
        logits.append(s.step(int(t)))
        traces.append(torch.stack(s.trace))
    return torch.stack(logits), torch.stack(traces, 1)


def tensor_shapes(cfg: dict) -> dict:
    """name -> shape of every tensor a checkpoint of this config holds."""
    W, V = cfg["width"], cfg["vocab"]
    sh = {"embed": (V, W), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W), "pos": (cfg["max_positions"], W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        q = p + "mix."
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        sh[p + "norm1"] = (W,)
        if L["type"] == "delta":
            G, taps = m.get("kv_heads", H), m["conv"]
            for n, c in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                sh[q + n], sh[q + n + ".conv"] = (c, W), (c, taps)
            sh.update({q + "b": (H, W), q + "a": (H, W), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (Dv,), q + "g": (H * Dv, W), q + "o": (W, H * Dv)})
        else:
            R = m["kv_rank"]
            sh[q + "q"] = (H * D, W)
            if m.get("kv_from") is None:
                sh[q + "dkv"], sh[q + "dkv.norm"] = (R, W), (R,)
            sh.update({q + "uk": (H * D, R), q + "uv": (H * Dv, R), q + "o": (W, H * Dv)})
        mlp = L.get("mlp")
        if mlp:
            F, f = mlp["expert"]["ff"], p + "mlp."
            sh[p + "norm2"] = (W,)
            sh[f + "router"] = (mlp["router"]["experts"], W)
            for e in range(mlp["router"]["experts"]):
                sh.update({"%se%d.gate" % (f, e): (F, W), "%se%d.up" % (f, e): (F, W), "%se%d.down" % (f, e): (W, F)})
            if mlp.get("shared"):
                Fs = mlp["shared"]["ff"]
                sh.update({f + "shared.gate": (Fs, W), f + "shared.up": (Fs, W), f + "shared.down": (W, Fs), f + "shared.sg": (1, W)})
    sh["final.norm"], sh["head"] = (W,), (V, W)
    return sh


def random_weights(cfg: dict, seed: int, router_spread: float = 2.0) -> dict:
    """bf16-representable random weights; the router's rows are spread so that choices are rarely close."""
    gen = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in name:
            t = 1.0 + 0.2 * torch.randn(shape, generator=gen)
        elif last == "A_log":
            t = torch.log(0.3 + 2.0 * torch.rand(shape, generator=gen))
        elif last == "dt_bias":
            t = torch.randn(shape, generator=gen) - 2.0
        elif last == "conv":
            t = 0.5 * torch.randn(shape, generator=gen)
        elif name in ("embed", "bigram", "pos"):
            t = torch.randn(shape, generator=gen) * (0.7 if name == "embed" else 0.4)
        elif last == "router":
            t = router_spread * torch.randn(shape, generator=gen) / math.sqrt(shape[-1])
        else:
            t = torch.randn(shape, generator=gen) / math.sqrt(shape[-1])
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w
