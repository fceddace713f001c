"""Models the engine serves, and what the engine asks of them.

`registry` maps a configuration to its model class and a model folder to its
configuration; `base.ServedModel` is the interface the engine drives.
"""
