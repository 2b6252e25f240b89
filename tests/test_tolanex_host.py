"""Host-side checks for the Tolanex family: the registry reads a model directory's config.json into the C structs (and the Python
mirror fills the same bytes), and the plain restatement the GPU tests lean on is itself checked mechanism by mechanism on
hand-made cases (no GPU)."""
import ctypes as C
import json
import math
from importlib import import_module

import torch

from oracle import tolanex_oracle as O

D = torch.float64


def small_cfg():
    d = {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 3, "conv": 3}
    l = {"heads": 2, "dim": 5, "vdim": 3, "kv_rank": 7, "scale": 0.3}
    moe = {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}, "scale": 2.5}, "shared": {"ff": 11}}
    return {"architecture": "Tolanex", "vocab": 31, "width": 12, "max_positions": 40, "residual_mult": 0.45, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": 17, "mul_prev": 5000000019, "mul_cur": 3}}, "layers": [
                {"type": "delta", "mixer": d, "mlp": moe},
                {"type": "latent_attention", "mixer": l, "mlp": None},
                {"type": "latent_attention", "mixer": dict(l, kv_from=1, heads=3, dim=4), "mlp": moe}]}


def read(lib, capi, cfg, path, room=8):
    (path / "config.json").write_text(json.dumps(cfg))
    c, specs = capi.b2_config(), (capi.b2_layer_spec * 8)()
    return lib.b2_config_from_dir(str(path).encode(), C.byref(c), specs, room), c, specs


def test_registry_reads_the_layer_list(pkg, lib, tmp_path):
    capi = import_module("aws-k8s-ansible-provisioner_b200.capi")
    eng = import_module("aws-k8s-ansible-provisioner_b200.engine")
    cfg = small_cfg()
    rc, c, specs = read(lib, capi, cfg, tmp_path)
    assert rc == 0, lib.b2_last_error()
    assert (c.arch, c.num_layers, c.hidden, c.vocab, c.norm_kind, c.tie_embeddings, c.max_positions) == (capi.ARCH_TOLANEX, 3, 12, 31, 2, 0, 40)
    assert (c.bigram_buckets, c.bigram_mul_prev, c.bigram_mul_cur) == (17, 5000000019, 3)
    assert abs(c.residual_mult - 0.45) < 1e-6 and abs(c.rms_eps - 1e-5) < 1e-11
    s0, s1, s2 = specs[0], specs[1], specs[2]
    assert (s0.mixer, s0.heads, s0.kv_heads, s0.dim, s0.vdim, s0.conv_taps, s0.kv_from) == (capi.MIXER_HEAD_DELTA, 4, 2, 5, 3, 3, -1)
    assert (s0.ff, s0.ff_dim, s0.experts, s0.top, s0.groups, s0.groups_keep, s0.shared_ff) == (capi.FF_SOFTMAX_EXPERTS, 9, 6, 2, 3, 2, 11)
    assert abs(s0.router_scale - 2.5) < 1e-6
    assert (s1.mixer, s1.heads, s1.dim, s1.rot_dim, s1.vdim, s1.kv_rank, s1.kv_from, s1.ff) == (capi.MIXER_LATENT_ATTENTION, 2, 5, 0, 3, 7, -1, capi.FF_NONE)
    assert abs(s1.scale - 0.3) < 1e-6
    assert (s2.mixer, s2.heads, s2.dim, s2.kv_from) == (capi.MIXER_LATENT_ATTENTION, 3, 4, 1)
    # the Python mirror fills the same bytes from the same dict, and reads them back into an equal layer list
    mine, again = (capi.b2_layer_spec * 3)(), (capi.b2_layer_spec * 3)()
    for sp, layer in zip(mine, cfg["layers"]):
        eng._fill_layer_spec(sp, dict(layer, _family="tolanex"))
    assert bytes(mine) == bytes(specs)[:C.sizeof(mine)]
    for sp, layer in zip(again, [eng._layer_dict(specs[i], "tolanex") for i in range(3)]):
        eng._fill_layer_spec(sp, dict(layer, _family="tolanex"))
    assert bytes(again) == bytes(mine)
    ec = eng.EngineConfig.tolanex(cfg)
    assert (ec.arch, ec.max_positions, ec.bigram, ec.norm_kind) == ("tolanex", 40, (17, 5000000019, 3), 2)


def test_registry_optional_keys_and_refusals(pkg, lib, tmp_path):
    capi = import_module("aws-k8s-ansible-provisioner_b200.capi")
    cfg = small_cfg()
    del cfg["residual_mult"], cfg["layers"][0]["mixer"]["kv_heads"]
    mlp = cfg["layers"][0]["mlp"]
    del mlp["shared"], mlp["router"]["groups"], mlp["router"]["scale"]
    rc, c, specs = read(lib, capi, cfg, tmp_path)
    assert rc == 0, lib.b2_last_error()
    assert c.residual_mult == 1.0
    assert (specs[0].kv_heads, specs[0].groups, specs[0].groups_keep, specs[0].shared_ff, specs[0].router_scale) == (4, 1, 1, 0, 1.0)
    for spoil, word in ((lambda k: k["layers"][0].update(type="delta_2"), b"delta_2"), (lambda k: k["embedding"].pop("bigram"), b"bigram"),
                        (lambda k: k.pop("max_positions"), b"max_positions"), (lambda k: k["layers"][0]["mlp"].update(kind="dense"), b"dense"),
                        (lambda k: k["layers"][1]["mixer"].pop("kv_rank"), b"kv_rank"), (lambda k: k["layers"][0]["mixer"].pop("conv"), b"conv")):
        bad = small_cfg()
        spoil(bad)
        assert read(lib, capi, bad, tmp_path)[0] != 0 and word in lib.b2_last_error(), word
    assert read(lib, capi, small_cfg(), tmp_path, room=2)[0] != 0


def test_bigram_rows_by_hand():
    assert O.bigram_row(None, 4, 17, 5, 3) == 17
    assert O.bigram_row(2, 4, 17, 5, 3) == (10 + 12) % 17
    assert O.bigram_row(30, 30, 17, 5000000019, 3) == (30 * 5000000019 + 90) % 17
    w = {"embed": torch.arange(10.0, dtype=D).view(5, 2), "bigram": 100 * torch.arange(8.0, dtype=D).view(4, 2), "pos": torch.full((6, 2), 0.5, dtype=D)}
    emb = {"bigram": {"buckets": 3, "mul_prev": 2, "mul_cur": 1}}
    assert torch.equal(O.embed(w, emb, None, 1, 0), torch.tensor([2.5 + 600, 3.5 + 700], dtype=D))
    assert torch.equal(O.embed(w, emb, 1, 2, 3), torch.tensor([4.5 + 200, 5.5 + 300], dtype=D))       # (2 + 2) mod 3 = 1


def test_output_norm_and_expert_by_hand():
    x = O.out_norm_add(torch.tensor([1.0, 1.0], dtype=D), torch.tensor([3.0, 4.0], dtype=D), torch.tensor([2.0, 1.0], dtype=D), 0.5, 0.0)
    r = math.sqrt(12.5)
    assert torch.allclose(x, torch.tensor([1 + 0.5 * 6 / r, 1 + 0.5 * 4 / r], dtype=D))
    w = {"e.gate": torch.tensor([[1.0, 0.0]], dtype=D), "e.up": torch.tensor([[0.0, 1.0]], dtype=D), "e.down": torch.tensor([[2.0], [1.0]], dtype=D)}
    g = 3.0 / (1 + math.exp(-3.0)) * -5.0
    assert torch.allclose(O.gated_expert(torch.tensor([3.0, -5.0], dtype=D), w, "e."), torch.tensor([2 * g, g], dtype=D))


def test_routing_by_hand():
    z = torch.tensor([3.0, -9.0, 2.0, 1.9, 0.5, 2.5], dtype=D)      # groups of two: best 3.0, 2.0, 2.5
    s = torch.softmax(z, 0)
    idx, wt = O.route(z, 3, 3, 2, 2.0)                              # the group {2, 3} is out although 2.0 and 1.9 are large (and their SUM is the largest)
    assert idx == [0, 5, 4] and torch.allclose(torch.stack(wt), 2.0 * s[idx])
    idx, wt = O.route(z, 3, 1, 1, 1.0)
    assert idx == [0, 5, 2] and torch.allclose(torch.stack(wt), s[idx])      # not renormalised
    assert O.route(torch.zeros(4, dtype=D), 2, 2, 1, 1.0)[0] == [0, 1]       # ties: the lower index


def test_delta_rule_by_hand():
    S = torch.tensor([[1.0, 2.0], [0.0, -1.0]], dtype=D)
    q, k, v = torch.tensor([1.0, 1.0], dtype=D), torch.tensor([0.6, 0.8], dtype=D), torch.tensor([3.0, -2.0], dtype=D)
    S1, o = O.delta_step(S, q, k, v, torch.tensor(0.5, dtype=D), torch.tensor(0.25, dtype=D))
    Sg = 0.5 * S
    u = 0.25 * (v - torch.tensor([0.6 * 0.5, 0.6 * 1.0 - 0.8 * 0.5], dtype=D))
    want = Sg + torch.outer(k, u)
    assert torch.allclose(S1, want) and torch.allclose(o, want.sum(0))       # the read-out sees the write
    # beta 1, no decay: the state returns v for k exactly
    S2, _ = O.delta_step(S, q, k, v, torch.tensor(1.0, dtype=D), torch.tensor(1.0, dtype=D))
    assert torch.allclose(S2.T @ k, v)
    g = O.head_decay(torch.tensor(0.3, dtype=D), torch.tensor(-0.2, dtype=D), torch.tensor(0.1, dtype=D))
    assert abs(float(g) - math.exp(-math.exp(-0.2) * math.log1p(math.exp(0.4)))) < 1e-12
    hist, y = O.conv_step(torch.tensor([[1.0], [2.0]], dtype=D), torch.tensor([3.0], dtype=D), torch.tensor([[10.0, 100.0, 1000.0]], dtype=D))
    assert float(y) == 10 + 200 + 3000 and hist.flatten().tolist() == [2.0, 3.0]


def test_latent_attention_by_hand_and_shared_latents():
    lat = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]], dtype=D)
    uk, uv = torch.tensor([[1.0, 2.0]], dtype=D), torch.tensor([[3.0, -1.0]], dtype=D)
    s = torch.tensor([1.0, 2.0, 3.0], dtype=D) * 0.7 * 0.5
    want = (torch.softmax(s, 0) * torch.tensor([3.0, -1.0, 2.0], dtype=D)).sum()
    assert torch.allclose(O.latent_attention_step(torch.tensor([0.7], dtype=D), lat, uk, uv, 1, 1, 1, 0.5), want[None])
    # a layer with kv_from depends on the named layer's down-projection and has none of its own
    cfg = small_cfg()
    w = O.random_weights(cfg, seed=5)
    assert "l2.mix.dkv" not in w and "l1.mix.dkv" in w
    toks = [3, 30, 7, 7, 1, 12]
    base, st = O.forward(cfg, w, toks)
    w2 = dict(w)
    w2["l1.mix.dkv"] = w["l1.mix.dkv"].flip(0)
    w2["l1.mix.o"] = torch.zeros_like(w["l1.mix.o"])      # layer 1 itself adds nothing: only layer 2 can tell the difference
    w3 = dict(w2, **{"l1.mix.dkv": w["l1.mix.dkv"]})
    assert (O.forward(cfg, w2, toks)[0] - O.forward(cfg, w3, toks)[0]).abs().max() > 1e-4


def test_whole_model_shapes_and_causality():
    cfg = small_cfg()
    weights = import_module("aws-k8s-ansible-provisioner_b200.weights")
    assert weights.tolanex_tensor_shapes(cfg) == O.tensor_shapes(cfg)
    sd = weights.tolanex_random_state_dict(cfg)
    assert {k: tuple(v.shape) for k, v in sd.items()} == O.tensor_shapes(cfg)
    w = O.random_weights(cfg, seed=6)
    toks = [3, 30, 7, 7, 1, 12, 25, 0, 9, 18, 4]
    logits, streams = O.forward(cfg, w, toks)
    assert streams.shape == (3, len(toks), 12) and logits.shape == (len(toks), 31) and torch.isfinite(logits).all()
    assert torch.allclose(O.forward(cfg, w, toks[:6])[0], logits[:6], atol=1e-12)
    assert O.Stepper(cfg, w).greedy(toks[:4], 3)[0] == int(torch.argmax(logits[3]))
    # the same token after another one is another input
    a, b = O.forward(cfg, w, [5, 7])[0][1], O.forward(cfg, w, [6, 7])[0][1]
    assert (a - b).abs().max() > 1e-4
