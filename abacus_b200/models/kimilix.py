"""The Kimilix decoder: its name in config.json and the names of its tensors.

Layer i's tensors start with "l<i>."; a mixer's are "l<i>.mix.*", a feed-forward's "l<i>.mlp.*" (expert e's
"l<i>.mlp.e<e>.*", the shared expert's "l<i>.mlp.shared.*"), the norms behind the mixer and the feed-forward "l<i>.norm1" and
"l<i>.norm2", their gains "l<i>.ls1" and "l<i>.ls2". The frame's are "embed", which is the output matrix too, and "final.norm".
"""
from ..config.kimilix import KimilixConfig
from ..config.registry import register_architecture
from .layout import ModelLayout
from .model import expected_tensors

_ATTENTION = {"wq": "q", "wk": "k", "wv": "v", "q_norm": "q.norm", "k_norm": "k.norm", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2",
              "lk2": "lk2", "wo": "o"}
_LATENT = {"wdq": "dq", "q_norm": "dq.norm", "wq": "uq", "wdown": "dkv", "down_norm": "dkv.norm", "wuk": "uk", "wuv": "uv",
           "wo": "o"}
_BY_KIND = {"attention": _ATTENTION, "latent_attention": _LATENT}
_SHARED = {"shared_gate_proj": "gate", "shared_up": "up", "shared_down": "down", "shared_gate": "sg"}


class KimilixArchitecture:
    name = "Kimilix"

    def parse_config(self, raw):
        return KimilixConfig.from_dict(raw)

    def layout(self, spec):
        layers = []
        for l, block in enumerate(spec.layers):
            p = f"l{l}."
            names = {("mixer_post_norm", "weight"): p + "norm1", ("mixer_post_norm", "gain"): p + "ls1"}
            for slot, short in _BY_KIND[block.mixer.kind].items():
                names[("mixer", slot)] = p + "mix." + short
            ffn = block.ffn
            if ffn is not None:
                names.update({("ffn_post_norm", "weight"): p + "norm2", ("ffn_post_norm", "gain"): p + "ls2"})
                if ffn.kind == "routed_mlp":
                    names.update({("ffn", "router"): p + "mlp.router", ("ffn", "router_bias"): p + "mlp.router.b"})
                    for e in range(ffn.experts):
                        for slot in ("gate", "up", "down"):
                            names[("ffn", f"{slot}{e}")] = f"{p}mlp.e{e}.{slot}"
                    for slot, short in _SHARED.items():
                        names[("ffn", slot)] = f"{p}mlp.shared.{short}"
                else:
                    for slot in ("up", "down"):
                        names[("ffn", slot)] = p + "mlp." + slot
            layers.append(names)
        return ModelLayout(embed="embed", final_norm="final.norm", head="head", layers=layers)

    def random_moments(self, name, shape, std, norm_std):
        """(mean, amplitude) of a random tensor of this design where the general rule (matrices around zero, vectors
        around one) does not fit; None: the general rule."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or name == "final.norm":  # stored around zero
            return 0.0, norm_std
        if last in ("lq1", "lk1", "lq2", "lk2"):
            return 0.0, 0.1
        if last == "b":
            return 0.0, 0.5
        return None

    def info(self, spec):
        kinds = "".join("a" if b.mixer.kind == "attention" else "l" for b in spec.layers)
        ffs = "".join("-" if b.ffn is None else "e" if b.ffn.kind == "routed_mlp" else "d" for b in spec.layers)
        return f"kimilix dim={spec.hidden} layers={len(spec.layers)} ({kinds}; feed-forwards {ffs}) vocab={spec.vocab}"

    def tensor_names(self, spec, available=None):
        return expected_tensors(spec, self.layout(spec), available)


register_architecture(KimilixArchitecture())
