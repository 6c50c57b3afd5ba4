"""models subpackage."""


def make_executor(weights, dtype: str = "bfloat16", **kw):
    """Executor class for the checkpoint's architecture.  ``dtype``: compute precision (``float32`` where the family
    declares it)."""
    from .registry import plugin_for
    arch = weights.config.arch
    if arch == "sisisun":
        from .sisisun import SisisunExecutor
        return SisisunExecutor(weights, dtype=dtype, **kw)
    if dtype != "bfloat16":
        raise ValueError(f"{arch}: compute dtype {dtype!r} is not built (supported: {plugin_for(arch).compute_dtypes})")
    if arch == "gemma4":
        from .gemma4 import Gemma4Executor
        return Gemma4Executor(weights, **kw)
    from .executor import HybridExecutor
    return HybridExecutor(weights, **kw)
