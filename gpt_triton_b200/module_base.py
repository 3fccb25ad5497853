"""What the model modules of this package share: derived-operand caching and the eval-only base class."""

from torch import nn

from . import kernels as K


class _OperandCache:
    """Derived operands (PackedWeight and friends) per parameter; rebuilt when the parameter is replaced, cast,
    moved or written in place.  The tag uses the Parameter's own ``_version``, which ``load_state_dict``,
    ``param.copy_`` and optimizer steps bump (``param.data`` is a fresh tensor object whose counter always reads 0,
    so it cannot serve).  Writes made *through* ``param.data`` (``param.data.mul_(2)``) bump no counter torch
    exposes: after such a write call ``refresh_operands()`` on the model."""

    def __init__(self):
        self._slots = {}

    def clear(self):
        self._slots.clear()

    @staticmethod
    def _tag(param):
        return (param.data_ptr(), param._version, param.dtype, param.device, tuple(param.shape))

    def derived(self, key, params, make):
        """`make()` cached under `key` until one of `params` changes."""
        tag = tuple(self._tag(p) for p in params)
        slot = self._slots.get(key)
        if slot is None or slot[0] != tag:
            slot = (tag, make())
            self._slots[key] = slot
        return slot[1]

    def __call__(self, param, weight_is_nk=False):
        return self.derived(("packed", id(param), weight_is_nk), (param,),
                            lambda: K.pack_weight(param.data.contiguous(), weight_is_nk=weight_is_nk))

    def folded(self, weight, ln_weight, ln_bias, bias):
        """FoldedWeight of `weight` with the LayerNorm (ln_weight, ln_bias) in front of it and `bias` behind."""
        return self.derived(("folded", id(weight)), (weight, ln_weight, ln_bias, bias),
                            lambda: K.fold_layer_norm(weight.data.contiguous(), ln_weight.data.contiguous(), ln_bias.data.contiguous(),
                                                      bias.data.contiguous()))


class _EvalOnly(nn.Module):
    def _check_eval(self):
        if self.training:
            raise NotImplementedError("libb200gpt implements the forward/eval path only: call .eval() first")

    def refresh_operands(self):
        """Drop every cached derived operand (packed weights) of this module and its children; the next forward
        rebuilds them from the parameters.  Needed only after writes through ``param.data``, which torch's version
        counters do not see; ``load_state_dict``, ``copy_``, casts and moves are noticed without it."""
        for m in self.modules():
            cache = getattr(m, "_operand", None)
            if isinstance(cache, _OperandCache):
                cache.clear()
