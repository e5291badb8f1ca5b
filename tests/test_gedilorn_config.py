"""Gedilorn without a GPU: its configuration (keys, defaults, faults, layers that use another layer's weights), the parts and
tensor names its builder picks, what the cache keeps, the prompt tables of its mixer, and the plain implementation's mechanisms
against the same sums written another way."""
import json
import math

import numpy as np
import pytest
import torch

from helpers import GEDILORN_CONFIGS, gedilorn_config, random_tokens, write_gedilorn
from plain import gedilorn_plain as P


def build(name):
    from rocmforge_b200.config import architecture_for
    return architecture_for("Gedilorn").build(gedilorn_config(GEDILORN_CONFIGS[name])[0])


def test_the_design_is_chosen_by_its_name(tmp_path):
    from rocmforge_b200.config import load_config
    write_gedilorn(GEDILORN_CONFIGS["GA"], str(tmp_path))
    arch, cfg = load_config(str(tmp_path))
    assert arch.name == "Gedilorn" and (cfg.width, cfg.vocab, cfg.eps, cfg.streams) == (64, 96, 1e-5, 2)
    assert (cfg.embedding_scale, cfg.logit_scale) == (3.0, 0.7)
    assert (cfg.pairs.buckets, cfg.pairs.mul_prev, cfg.pairs.mul_cur) == (37, 1009, 53)
    assert [L.type for L in cfg.layers] == ["latent_attention_2", "latent_attention", "latent_attention_2", "latent_attention_2"]
    assert [L.weights_of for L in cfg.layers] == [None, None, 0, 0] and [L.ff for L in cfg.layers] == [40, None, 40, 40]
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.rot_base, m.gated) == (3, 10, 6, 14, 21, 0.3, 50.0, True)
    assert m.rot_scaling == dict(factor=3.0, original=24.0, fast=4.0, slow=1.0)
    assert (cfg.layers[1].mixer.rot_dim, cfg.layers[1].mixer.rot_base, cfg.layers[1].mixer.gated) == (0, None, False)
    written = json.load(open(tmp_path / "config.json"))
    assert {k: v for k, v in cfg.to_dict().items() if k != "torch_dtype"} == {k: v for k, v in written.items() if k != "torch_dtype"}


def test_what_a_configuration_may_leave_out():
    cfg, _ = gedilorn_config(GEDILORN_CONFIGS["GB"])
    assert cfg.streams is None and cfg.pairs is None and cfg.logit_scale == 1.0 and cfg.layers[0].mixer.rot_scaling is None
    cfg, _ = gedilorn_config(GEDILORN_CONFIGS["GD"])
    assert cfg.embedding_scale == 1.0 and cfg.pairs.buckets == 1


@pytest.mark.parametrize("path,value,error", [
    ("width", None, "MissingKey"), ("vocab", 0, "InvalidValue"), ("norm.eps", None, "MissingKey"), ("layers", [], "InvalidValue"),
    ("streams", 0, "InvalidValue"), ("embedding.bigram.buckets", 0, "InvalidValue"), ("embedding.bigram.mul_cur", None, "MissingKey"),
    ("embedding.bigram.mul_prev", 0.5, "InvalidValue"), ("logit_scale", "x", "InvalidValue"),
    ("layers.0.type", "attention", "InvalidValue"), ("layers.0.mixer.heads", 0, "InvalidValue"), ("layers.0.mixer.dim", None, "MissingKey"),
    ("layers.0.mixer.kv_rank", 0, "InvalidValue"), ("layers.0.mixer.vdim", None, "MissingKey"), ("layers.0.mixer.scale", 0, "InvalidValue"),
    ("layers.0.mixer.rot_dim", 7, "InvalidValue"), ("layers.0.mixer.rot.dims", 4, "InvalidValue"), ("layers.0.mixer.rot.base", 1.0, "InvalidValue"),
    ("layers.0.mixer.rot.scaling.slow", None, "MissingKey"), ("layers.0.mlp.kind", "moe", "InvalidValue"), ("layers.0.mlp.ff", None, "MissingKey"),
    ("layers.2.weights_of", 2, "InvalidValue"), ("layers.2.weights_of", 9, "InvalidValue"), ("layers.2.weights_of", 1, "InvalidValue"),
    ("layers.2.mixer.scale", 0.4, "InvalidValue"), ("layers.2.mlp.ff", 48, "InvalidValue"), ("layers.0.weights_of", 3, "InvalidValue"),
])
def test_faults_of_a_configuration_name_their_key(path, value, error):
    from rocmforge_b200.config import architecture_for, errors
    raw = json.loads(json.dumps(gedilorn_config(GEDILORN_CONFIGS["GA"])[1]))       # layers that share nothing
    cur, parts = raw, path.split(".")
    for p in parts[:-1]:
        cur = cur[int(p)] if p.isdigit() else cur[p]
    last = int(parts[-1]) if parts[-1].isdigit() else parts[-1]
    if value is None:
        del cur[last]
    else:
        cur[last] = value
    with pytest.raises(getattr(errors, error)) as e:
        architecture_for("Gedilorn").config_cls.from_dict(raw)
    # two layers that should be equal and are not: the fault is named where they meet
    met = "weights_of" if path in ("layers.2.mixer.scale", "layers.2.mlp.ff", "layers.0.weights_of") else parts[-1]
    assert met in str(e.value)


@pytest.mark.parametrize("name", list(GEDILORN_CONFIGS))
def test_tensor_names_shapes_and_what_the_cache_keeps(name):
    from rocmforge_b200.cache.requests import KVRequest, StateRequest
    from rocmforge_b200.engine.model import EMBEDDING
    c = GEDILORN_CONFIGS[name]
    spec = build(name)
    specs, W, S = spec.param_specs(), c["width"], c.get("streams")
    want = {"embed": (c["vocab"], W), "embed.norm": (W,), "final.norm": (W,), "head": (c["vocab"], W)}
    pairs = c.get("embedding", {}).get("bigram")
    if pairs:
        want["bigram"] = (pairs["buckets"] + 1, W)
    for i, L in enumerate(c["layers"]):
        if "weights_of" in L:
            continue
        m, p = L["mixer"], f"l{i}."
        hq = m["heads"] * (m["dim"] + m["rot_dim"])
        want.update({p + "norm1": (W,), p + "mix.q": (hq, W), p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], W), p + "mix.dkv.norm": (m["kv_rank"],),
                     p + "mix.uk": (m["heads"] * m["dim"], m["kv_rank"]), p + "mix.uv": (m["heads"] * m["vdim"], m["kv_rank"]),
                     p + "mix.o": (W, m["heads"] * m["vdim"])})
        if L["type"] == "latent_attention_2":
            want[p + "mix.g"] = (m["heads"] * m["vdim"], W)
        if L["mlp"]:
            want.update({p + "norm2": (W,), p + "mlp.gate": (L["mlp"]["ff"], W), p + "mlp.up": (L["mlp"]["ff"], W), p + "mlp.down": (W, L["mlp"]["ff"])})
        for q in (1, 2) if S else ():
            if q == 1 or L["mlp"]:
                want.update({f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
    assert {k: s.shape for k, s in specs.items() if not s.optional} == want
    requests = spec.cache_requests()
    assert requests[EMBEDDING] == (StateRequest((("last", (2,), torch.int32),), repeatable=True) if pairs else None)
    assert len(spec.schedule) == len(c["layers"]) and len(spec.blocks) == sum("weights_of" not in L for L in c["layers"])
    for i, L in enumerate(c["layers"]):
        owner = L.get("weights_of", i)
        assert spec.block_prefixes[spec.schedule[i].layer] == f"l{owner}." and spec.schedule[i].kv_from is None
        m = L["mixer"]
        row = -(-(m["kv_rank"] + m["rot_dim"]) // 8) * 8
        assert requests[i] == KVRequest(1, row, v_head_dim=m["kv_rank"], values_are_keys=True)       # every run has rows of its own


def test_a_layer_without_feed_forward_may_store_what_it_does_not_use(tmp_path):
    from rocmforge_b200.weights.loader import check_folder
    from rocmforge_b200.weights.safetensors_io import ModelFiles
    write_gedilorn(GEDILORN_CONFIGS["GA"], str(tmp_path))
    specs = build("GA").param_specs()
    check_folder(ModelFiles(str(tmp_path)), specs)
    assert {k for k, s in specs.items() if s.optional} == {"l1.norm2", "l1.hc2.in", "l1.hc2.out", "l1.hc2.mix"}


def test_rows_hold_keys_and_values_at_once():
    """One plane of rows for keys and values: the values are a view of the rows' first numbers."""
    from rocmforge_b200.cache import SequenceCache
    from rocmforge_b200.cache.requests import KVRequest, StateRequest
    req = KVRequest(1, 40, v_head_dim=24, values_are_keys=True)
    state = StateRequest((("last", (2,), torch.int32),), repeatable=True)
    cache = SequenceCache({-1: state, 0: req, 1: req}, max_tokens=256, max_slots=2, dtype=torch.float32)
    v = cache.view(1)
    assert v.k_pages.shape == (4, 1, 64, 40) and v.v_pages.shape == (4, 1, 64, 24) and v.k_pages.data_ptr() == v.v_pages.data_ptr()
    assert len(cache.groups) == 1 and cache.groups[0].storage.numel() == 2 * 4 * 64 * 40 and cache.groups[0].value_storage is None
    assert cache.view(-1)["last"].shape == (2, 2) and cache.steps_repeatable
    cache = SequenceCache({0: StateRequest.of(S=(2, 3))}, max_tokens=64, max_slots=2, dtype=torch.float32)
    assert not cache.steps_repeatable
    with pytest.raises(ValueError):
        KVRequest(1, 16, v_head_dim=17, values_are_keys=True)


def test_the_prompt_tables_of_the_mixer():
    from rocmforge_b200 import StepRequest
    from rocmforge_b200.engine.batch import StepBatch
    mixer = build("GC").blocks[0].mixer
    batch = StepBatch([StepRequest(0, [1] * 300), StepRequest(1, [1] * 5), StepRequest(2, [1] * 129)], [0, 700, 64], 10)
    tiles = mixer.step_table("attention_tiles128", batch).reshape(-1, 2).tolist()
    assert sorted(map(tuple, tiles)) == [(0, 0), (0, 128), (0, 256), (1, 0), (2, 0), (2, 128)]
    keys = [[0, 700, 64][i] + r for i, r in tiles]
    assert keys == sorted(keys)
    assert mixer.step_table("context_rows", batch).tolist() == [0, 300, 1005, 1198]
    one = StepBatch([StepRequest(0, [1]), StepRequest(1, [1])], [3, 9], 10)
    assert mixer.step_table("context_rows", one).size == 0 and mixer.step_table("attention_tiles128", one).size == 0


# --------------------------------------------------------------------------- the plain implementation against closed forms

def test_plain_rows_of_pairs():
    assert P.pair_rows([4], 3, 5, 7) == [7]
    assert P.pair_rows([4, 6, 4], 3, 5, 7) == [7, (12 + 30) % 7, (18 + 20) % 7]


def test_plain_streams_from_to():
    """Two streams, one column: a mix that sends stream 0 to stream 1 and nothing back."""
    xs = torch.tensor([[[2.0]], [[3.0]]])
    mix = torch.tensor([[0.0, 1.0], [0.0, 0.0]])
    new = P.spread(xs, mix, torch.tensor([10.0, 100.0]), torch.tensor([[1.0]]))
    assert new[:, 0, 0].tolist() == [10.0, 102.0] and float(P.collect(xs, torch.tensor([1.0, -1.0]))) == -1.0


def test_plain_rotation_turns_neighbours_and_lengthens():
    f, mag = P.stretched_frequencies(4, 100.0, None)
    assert mag == 1.0 and torch.allclose(f, torch.tensor([1.0, 0.1], dtype=torch.float64))
    x = torch.tensor([[1.0, 0.0, 0.0, 1.0]], dtype=torch.float64)
    y = P.turn_neighbours(x, torch.tensor([2]), f, 1.5)
    want = [1.5 * math.cos(2), 1.5 * math.sin(2), -1.5 * math.sin(0.2), 1.5 * math.cos(0.2)]
    assert torch.allclose(y[0], torch.tensor(want, dtype=torch.float64))
    from rocmforge_b200.parts import POSITIONS
    for dims, base, s in ((64, 1e6, (8.0, 8192, 32.0, 1.0)), (6, 50.0, (3.0, 24, 4.0, 1.0)), (16, 1e4, (2.0, 64, 8.0, 0.5))):
        sc = dict(zip(("factor", "original", "fast", "slow"), s))
        f, mag = P.stretched_frequencies(dims, base, sc)
        enc = POSITIONS.build("rope_yarn", head_dim=dims, theta=base, interleaved=True, **sc)
        assert np.allclose(enc.inv_freq_host.double(), f, rtol=1e-6) and abs(enc.magnitude - mag) < 1e-12
        assert enc.rotation()["interleaved"] and enc.rotation()["rot_dim"] == dims


def test_plain_attention_in_the_latents_space():
    """Folding W_uk into the queries and W_uv out of the result gives what expanding keys and values gives."""
    torch.manual_seed(0)
    m = dict(heads=3, dim=4, rot_dim=2, vdim=5, kv_rank=7, scale=0.4, rot=dict(dims=2, base=10.0))
    W = {"q": torch.randn(18, 6), "dkv": torch.randn(9, 6), "dkv.norm": torch.randn(7), "uk": torch.randn(12, 7), "uv": torch.randn(15, 7),
         "o": torch.randn(6, 15)}
    W = {k: v.double() for k, v in W.items()}
    h = torch.randn(9, 6, dtype=torch.float64)
    want = P.latent_attention(h, W, "", m, 1e-6)
    down = h @ W["dkv"].T
    c = P.rms_norm(down[:, :7], W["dkv.norm"], 1e-6)
    f, mag = P.stretched_frequencies(2, 10.0, None)
    r = P.turn_neighbours(down[:, 7:], torch.arange(9), f, mag)
    q = (h @ W["q"].T).view(9, 3, 6)
    qr = P.turn_neighbours(q[..., 4:], torch.arange(9), f, mag)
    outs = []
    for n in range(3):
        folded = torch.cat([q[:, n, :4] @ W["uk"].view(3, 4, 7)[n], qr[:, n]], dim=1)
        p = P.causal_softmax(folded @ torch.cat([c, r], dim=1).T * 0.4)
        outs.append((p @ c) @ W["uv"].view(3, 5, 7)[n].T)
    assert torch.allclose(torch.cat(outs, dim=1) @ W["o"].T, want)


def test_plain_model_sees_its_whole_past(tmp_path):
    """Changing the first token changes every later row; changing the last one changes no earlier row."""
    from safetensors.torch import load_file
    write_gedilorn(GEDILORN_CONFIGS["GA"], str(tmp_path))
    m = P.PlainGedilorn(json.load(open(tmp_path / "config.json")), load_file(str(tmp_path / "model.safetensors")))
    t = random_tokens(96, 12, 5)
    a = m.logits(t)
    b = m.logits([(t[0] + 1) % 96] + t[1:])
    c = m.logits(t[:-1] + [(t[-1] + 1) % 96])
    assert ((a - b).abs().amax(dim=1) > 1e-6).all() and torch.equal(a[:-1], c[:-1]) and (a[-1] - c[-1]).abs().max() > 1e-3
