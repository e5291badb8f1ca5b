"""Dubodra without a GPU: its configuration (keys, defaults, faults), the parts and tensor names its builder picks, what the
cache keeps per layer, and the plain implementation's mechanisms against the same sums written another way."""
import copy
import json
import math

import pytest
import torch

from helpers import DUBODRA_CONFIGS, dubodra_config, random_tokens, write_dubodra
from plain import dubodra_plain as P


def test_the_design_is_chosen_by_its_name(tmp_path):
    from rocmforge_b200.config import load_config
    write_dubodra(DUBODRA_CONFIGS["DA"], str(tmp_path))
    arch, cfg = load_config(str(tmp_path))
    assert arch.name == "Dubodra" and cfg.width == 64 and cfg.vocab == 96 and cfg.eps == 1e-5
    assert cfg.embedding_scale == 2.0 and cfg.logit_softcap == 8.0 and cfg.side_dim == 5
    assert [L.type for L in cfg.layers] == ["delta", "attention", "lightning", "attention"]
    d, a, n = (L.mixer for L in cfg.layers[:3])
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.taps) == (4, 2, 24, 12, 3)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.rot_dims, a.rot_base) == (4, 2, 16, 24, 0.4, 5.0, 8, 100.0)
    assert (n.heads, n.dim, n.vdim, n.decay) == (2, 24, 12, [0.5, 1.0])
    f = cfg.layers[0].mlp
    assert (f.kind, f.experts, f.identity, f.top, f.scale, f.groups, f.keep) == ("moe", 5, 1, 2, 1.7, 3, 2)
    assert (f.expert.ff, f.expert.limit, f.shared.ff, f.shared.limit) == (20, 0.7, 24, 1.2)
    assert cfg.layers[1].mlp is None and (cfg.layers[2].mlp.kind, cfg.layers[2].mlp.ff) == ("dense", 40)
    assert cfg.to_dict() == json.load(open(tmp_path / "config.json"))


def test_what_a_configuration_may_leave_out():
    cfg, _ = dubodra_config(DUBODRA_CONFIGS["DB"])
    assert cfg.embedding_scale == 1.0 and cfg.logit_softcap is None and cfg.side_dim is None
    cfg, _ = dubodra_config(DUBODRA_CONFIGS["DA"])
    a, f = cfg.layers[3].mixer, cfg.layers[3].mlp
    assert a.softcap is None and a.rot_dims == 0 and a.rot_base is None
    assert (f.scale, f.identity, f.groups, f.keep, f.shared) == (1.0, 0, 1, 1, None)


@pytest.mark.parametrize("path,value,error", [
    ("width", None, "MissingKey"), ("vocab", 0, "InvalidValue"), ("norm.eps", None, "MissingKey"), ("layers", [], "InvalidValue"),
    ("token_side.dim", None, "MissingKey"), ("token_side.dim", 0, "InvalidValue"), ("logit_softcap", 0.0, "InvalidValue"),
    ("layers.0.type", "mamba2", "InvalidValue"), ("layers.0.mixer.kv_heads", 3, "InvalidValue"), ("layers.0.mixer.conv", 17, "InvalidValue"),
    ("layers.0.mixer.dim", 257, "InvalidValue"), ("layers.0.mixer.vdim", None, "MissingKey"),
    ("layers.0.mlp.kind", "glu", "InvalidValue"), ("layers.0.mlp.expert.limit", None, "MissingKey"), ("layers.0.mlp.expert.limit", 0, "InvalidValue"),
    ("layers.0.mlp.router.top", 7, "InvalidValue"), ("layers.0.mlp.router.groups.count", 4, "InvalidValue"),
    ("layers.0.mlp.router.groups.keep", 4, "InvalidValue"), ("layers.0.mlp.router.groups.keep", None, "MissingKey"),
    ("layers.0.mlp.shared.ff", None, "MissingKey"), ("layers.1.mixer.scale", None, "MissingKey"), ("layers.1.mixer.softcap", -1.0, "InvalidValue"),
    ("layers.1.mixer.rot.dims", 7, "InvalidValue"), ("layers.1.mixer.rot.dims", 18, "InvalidValue"), ("layers.1.mixer.rot.base", None, "MissingKey"),
    ("layers.2.mixer.decay", [0.5], "InvalidValue"), ("layers.2.mixer.decay", [0.5, 1.5], "InvalidValue"), ("layers.2.mixer.decay", None, "MissingKey"),
    ("layers.2.mixer.dim", 257, "InvalidValue"), ("layers.2.mlp.ff", None, "MissingKey"),
])
def test_faults_of_a_configuration_name_their_key(path, value, error):
    from rocmforge_b200.config import architecture_for, errors
    raw = copy.deepcopy(dubodra_config(DUBODRA_CONFIGS["DA"])[1])
    cur = raw
    parts = path.split(".")
    for p in parts[:-1]:
        cur = cur[int(p)] if p.isdigit() else cur[p]
    if value is None:
        del cur[parts[-1]]
    else:
        cur[parts[-1]] = value
    with pytest.raises(getattr(errors, error)) as e:
        architecture_for("Dubodra").config_cls.from_dict(raw)
    assert parts[-1] in str(e.value)


def test_too_few_experts_in_the_kept_groups():
    from rocmforge_b200.config import architecture_for, errors
    raw = copy.deepcopy(dubodra_config(DUBODRA_CONFIGS["DA"])[1])
    raw["layers"][0]["mlp"]["router"].update(top=3, groups={"count": 3, "keep": 1})
    with pytest.raises(errors.InvalidValue, match="keep"):
        architecture_for("Dubodra").config_cls.from_dict(raw)


def test_the_builder_picks_parts_and_names_by_the_configuration():
    from rocmforge_b200.config import architecture_for
    from rocmforge_b200.cache.requests import KVRequest, StateRequest
    for name, c in DUBODRA_CONFIGS.items():
        cfg, _ = dubodra_config(c)
        spec = architecture_for("Dubodra").build(cfg)
        specs = spec.param_specs()
        W, side = c["width"], (c.get("token_side") or {}).get("dim")
        want = {"embed": (c["vocab"], W), "head": (c["vocab"], W), "final.norm": (W,), "final.norm.b": (W,)}
        if side:
            want["side.embed"] = (c["vocab"], side * len(c["layers"]))
        requests = spec.cache_requests()
        for i, L in enumerate(c["layers"]):
            m, mlp, p = L["mixer"], L["mlp"], f"l{i}."
            want.update({p + "norm1": (W,), p + "norm1.b": (W,)})
            if mlp is None:
                assert specs[p + "norm2"].optional and specs[p + "norm2.b"].optional
            else:
                want.update({p + "norm2": (W,), p + "norm2.b": (W,)})
            H, D, V = m["heads"], m["dim"], m["vdim"]
            G = m.get("kv_heads", H)
            x = p + "mix."
            want[x + "o"] = (W, H * V)
            if L["type"] == "attention":
                want.update({x + "q": (H * D, W), x + "k": (G * D, W), x + "v": (G * V, W), x + "q.norm": (D,), x + "k.norm": (D,)})
                r = requests[i]
                assert isinstance(r, KVRequest) and (r.n_kv_heads, r.head_dim, r.window, r.chunk) == (G, D, None, None)
                assert (r.v_head_dim or r.head_dim) == V
            elif L["type"] == "lightning":
                want.update({x + "q": (H * D, W), x + "k": (H * D, W), x + "v": (H * V, W), x + "g": (H * V, W), x + "norm": (H * V,)})
                assert [(n, s, d) for n, s, d in requests[i].tensors] == [("S", (H, V, D), torch.float32)]
            else:
                want.update({x + "q": (G * D, W), x + "k": (G * D, W), x + "v": (H * V, W), x + "q.conv": (G * D, m["conv"]),
                             x + "k.conv": (G * D, m["conv"]), x + "v.conv": (H * V, m["conv"]), x + "b": (H, W), x + "a": (H, W),
                             x + "A_log": (H,), x + "dt_bias": (H,), x + "norm": (V,), x + "g": (H * V, W)})
                assert isinstance(requests[i], StateRequest)
                kept = {n: (s, d) for n, s, d in requests[i].tensors}
                assert kept.pop("S") == ((H, D, V), torch.float32)
                assert kept == ({"conv": ((m["conv"] - 1, 2 * G * D + H * V), torch.float32)} if m["conv"] > 1 else {})
            if side:
                want.update({p + "side.gate": (side, W), p + "side.proj": (W, side), p + "side.norm": (W,)})
            if mlp is not None and mlp["kind"] == "dense":
                want.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
            elif mlp is not None:
                E, ff, n = mlp["router"]["experts"], mlp["expert"]["ff"], mlp["router"].get("identity", 0)
                want.update({p + "mlp.router": (E + n, W), p + "mlp.correction": (E + n,)})
                for e in range(E):
                    want.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
                if "shared" in mlp:
                    s = mlp["shared"]["ff"]
                    want.update({p + "mlp.shared.gate": (s, W), p + "mlp.shared.up": (s, W), p + "mlp.shared.down": (W, s), p + "mlp.shared.sg": (1, W)})
        assert {k: tuple(v.shape) for k, v in specs.items() if not v.optional} == want, name
        assert specs["head"].tied_to is None and not spec.stop_token_ids


def test_only_the_modules_of_its_parts_are_compiled():
    from rocmforge_b200.config import architecture_for
    spec = architecture_for("Dubodra").build(dubodra_config(DUBODRA_CONFIGS["DC"])[0])
    assert set(spec.cuda_modules(torch.float32)) == {"gemm_simt", "sampling", "elementwise", "layernorm", "attention_generic", "retention",
                                                     "moe", "mamba2", "delta"}
    assert {"attention_prefill_tc", "attention_decode", "gemm_tcgen05"} <= set(spec.cuda_modules(torch.bfloat16))
    assert "attention_prefill" in spec.cuda_modules(torch.bfloat16)      # (one of its layers has no cap)


def test_parts_refuse_what_they_cannot_do():
    from rocmforge_b200.parts import FEED_FORWARDS, MIXERS
    base = dict(hidden=16, intermediate=8, n_experts=6, top=2, router_bias=False, activation="clamped_glu", limit=1.0)
    for bad in (dict(identity=1), dict(grouped=dict(groups=4, keep=1, scale=1.0)), dict(grouped=dict(groups=6, keep=1, scale=1.0)),
                dict(token_gate="sg"), dict(grouped=dict(groups=1, keep=1, scale=1.0), weight_on="input")):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build("routed_experts", **dict(base, **bad))
    FEED_FORWARDS.build("routed_experts", **base, grouped=dict(groups=2, keep=1, scale=1.0), identity=2, token_gate="sg")
    with pytest.raises(ValueError):
        FEED_FORWARDS.build("gated_mlp", hidden=16, intermediate=8, activation="clamped_glu")
    with pytest.raises(ValueError):
        MIXERS.build("retention", hidden=16, n_heads=1, dim=8, vdim=8, decay=[0.5], eps=1e-6, activation="silu", k_scale=0.5)
    with pytest.raises(ValueError):
        MIXERS.build("retention", hidden=16, n_heads=1, dim=300, vdim=8, decay=[0.5], eps=1e-6)
    with pytest.raises(ValueError):
        MIXERS.build("gated_delta", hidden=16, n_heads=2, qk_heads=1, dim=8, vdim=8, taps=2, decay_rank=None, gate_rank=None, eps=1e-6, gate_fn="relu")


# --------------------------------------------------------------------------- the plain mechanisms in another form

def test_plain_recurrences_as_sums_over_pairs():
    torch.manual_seed(0)
    T, D, V = 12, 5, 3
    q, k, v = torch.randn(T, D).double(), torch.randn(T, D).double(), torch.randn(T, V).double()
    o, S = P.fixed_decay_recurrence(q, k, v, 0.7)
    for t in range(T):
        want = sum(0.7 ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1))
        assert torch.allclose(o[t], want)
    a, S1 = P.fixed_decay_recurrence(q[:5], k[:5], v[:5], 0.7)
    b, S2 = P.fixed_decay_recurrence(q[5:], k[5:], v[5:], 0.7, S1)
    assert torch.allclose(torch.cat([a, b]), o) and torch.allclose(S2, S)
    # the corrected memory: with beta 1, decay 1 and unit keys it returns exactly what was last stored under a key
    kn = P.unit_vector(k)
    o, _ = P.corrected_recurrence(kn, kn, v, torch.ones(T).double(), torch.ones(T).double())
    assert torch.allclose(o, v, atol=1e-5)
    # and with beta 0 nothing is ever stored
    assert not P.corrected_recurrence(q, kn, v, torch.zeros(T).double(), torch.ones(T).double())[0].any()


def test_plain_short_functions():
    x = torch.linspace(-4, 4, 41).double()
    assert torch.allclose(P.gelu_by_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))
    h, W = torch.randn(6, 9).double() + 2.0, {"n": torch.randn(9).double(), "n.b": torch.randn(9).double()}
    assert torch.allclose(P.layer_norm(h, W, "n", 1e-5), torch.nn.functional.layer_norm(h, (9,), W["n"], W["n.b"], 1e-5))
    y = torch.randn(3, 2, 8).double()
    turned = P.turn_pairs(y, torch.tensor([0, 1, 7]), 4, 50.0)
    assert torch.equal(turned[0], y[0]) and torch.equal(turned[..., 4:], y[..., 4:])
    c, s = math.cos(7.0 * 50.0 ** -0.5), math.sin(7.0 * 50.0 ** -0.5)
    assert torch.allclose(turned[2, :, 1], y[2, :, 1] * c - y[2, :, 3] * s) and torch.allclose(turned[2, :, 3], y[2, :, 3] * c + y[2, :, 1] * s)
    u, w = torch.randn(5, 2).double(), torch.randn(2, 3).double()
    got = P.causal_taps(u, w)
    padded = torch.cat([torch.zeros(2, 2).double(), u])
    assert torch.allclose(got[3], P.silu((padded[3:6] * w.T).sum(0)))


def test_plain_groups():
    c = torch.tensor([[-0.1, -5.0, -0.2, -0.21, -4.0, 0.3]]).double()
    kept = P.limit_to_groups(c, 3, 2)
    assert kept.tolist()[0][2:4] == [float("-inf")] * 2 and kept[0, [0, 1, 4, 5]].tolist() == c[0, [0, 1, 4, 5]].tolist()
    assert math.isclose(float(P.choice_margin(c, 2, {"count": 3, "keep": 2})), 0.1, rel_tol=1e-6)      # the groups' gap: -0.1 against -0.2
    assert math.isclose(float(P.choice_margin(c, 2, None)), 0.1, rel_tol=1e-6)


def _mistakes():
    """name -> (what to replace in the plain module, the mistaken form, a configuration that has the mechanism)."""
    def no_correction(h, W, pre):
        s = torch.softmax(h @ W[pre + "router"].T, dim=-1)
        return s, s

    def closed_groups_count_as_zero(c, count, keep):
        return torch.nan_to_num(limit(c, count, keep), neginf=0.0)

    def group_by_sum(c, count, keep):
        g = c.view(c.shape[0], count, -1)
        best = g.sum(dim=-1).topk(keep, dim=-1).indices
        open_ = torch.zeros(c.shape[0], count, dtype=torch.bool).scatter_(1, best, True)
        return g.masked_fill(~open_[:, :, None], float("-inf")).reshape(c.shape)

    def unlimited(h, W, pre, cap):
        return clamped(h, W, pre, 1e9)

    def rms_instead(x, W, name, eps):
        return P.unit_rms(x, eps) * W[name] + W[name + ".b"]

    def read_before_write(q, k, v, beta, g, S=None):
        S = q.new_zeros((q.shape[1], v.shape[1]))
        out = []
        for t in range(q.shape[0]):
            S = g[t] * S
            out.append(S.T @ q[t])
            S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        return torch.stack(out), S

    def uncorrected(q, k, v, beta, g, S=None):
        S = q.new_zeros((q.shape[1], v.shape[1]))
        out = []
        for t in range(q.shape[0]):
            S = g[t] * S + torch.outer(k[t], beta[t] * v[t])
            out.append(S.T @ q[t])
        return torch.stack(out), S

    def decay_late(q, k, v, decay, S=None):
        o, S = fixed(q, k, v, decay)
        return o * decay, S

    def taps_reversed(x, w):
        return taps(x, w.flip(1))

    limit, clamped, fixed, taps, turn = P.limit_to_groups, P.clamped_unit, P.fixed_decay_recurrence, P.causal_taps, P.turn_pairs
    return {"no_correction": ("scores", no_correction, "DA"), "closed_groups_as_zero": ("limit_to_groups", closed_groups_count_as_zero, "DA"),
            "group_by_sum": ("limit_to_groups", group_by_sum, "DA"), "unlimited": ("clamped_unit", unlimited, "DA"),
            "rms_instead": ("layer_norm", rms_instead, "DB"), "read_before_write": ("corrected_recurrence", read_before_write, "DA"),
            "uncorrected": ("corrected_recurrence", uncorrected, "DA"), "decay_late": ("fixed_decay_recurrence", decay_late, "DC"),
            "taps_reversed": ("causal_taps", taps_reversed, "DD"), "relu_for_gelu": ("gelu_by_tanh", torch.relu, "DA"),
            "no_rotation": ("turn_pairs", lambda x, *a: x, "DB"), "slower_rotation": ("turn_pairs", lambda x, p, d, b: turn(x, p * 0.7, d, b), "DB"),
            "no_cap": ("capped", lambda z, cap: z, "DA"), "no_side_norm": ("token_side_input", lambda x, e, W, pre, eps: torch.zeros_like(x), "DD")}


@pytest.mark.parametrize("name", sorted(_mistakes()))
def test_a_mistake_in_any_mechanism_shows_in_the_logits(name, tmp_path, monkeypatch):
    """The test models are worth comparing with only if a mistaken mechanism moves their logits well beyond the bounds the
    engine is held to (3e-4 of the logits' spread in 32-bit, 2.5 % on average in bfloat16)."""
    from safetensors.torch import load_file
    what, wrong, model = _mistakes()[name]
    write_dubodra(DUBODRA_CONFIGS[model], str(tmp_path))
    m = P.PlainDubodra(json.load(open(tmp_path / "config.json")), load_file(str(tmp_path / "model.safetensors")))
    toks = random_tokens(DUBODRA_CONFIGS[model]["vocab"], 60, 5)
    right = m.logits(toks)
    monkeypatch.setattr(P, what, wrong)
    err = (m.logits(toks) - right).pow(2).mean(dim=-1).sqrt() / right.pow(2).mean().sqrt()
    assert float(err.mean()) > 0.03, f"{name}: only {float(err.mean()):.4f}"
